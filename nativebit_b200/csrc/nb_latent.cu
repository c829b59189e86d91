// Latent attention: keys and values of all heads are linear maps of one cached latent per position, plus one rotated key
// part that the heads share; a query sees a sliding window of positions.
//
//   nb_latent_prepare     norms the query latent and the key/value latent, rotates the shared key part, writes the cache
//   nb_latent_attention   a portion of a prompt: up-projected keys and values, online softmax (bf16: tensor cores, fp32:
//                         multiply-adds)
//   nb_latent_decode      one position per sequence, entirely in latent space: the query is taken through W_uk^T once, so
//                         the cached latents serve every head as keys and as values
#include <cuda_runtime.h>
#include <cuda_bf16.h>
#include <cooperative_groups.h>

#include <algorithm>
#include <cfloat>

#include "nb_layered.cuh"
#include "nb_mma.cuh"

namespace nb {

namespace cg = cooperative_groups;

// Element d of a rotated vector: pairs (2i, 2i + 1), (u, v) -> (u cos - v sin, v cos + u sin).  c, s: the position's rows
// of the tables, every pair's entry twice.
template <typename Get> __device__ __forceinline__ float rotated(Get x, const float* __restrict__ c, const float* __restrict__ s, int d) {
  return x(d) * c[d] + ((d & 1) ? x(d ^ 1) : -x(d ^ 1)) * s[d];
}

constexpr int kPrepThreads = 128, kPrepWarps = kPrepThreads / 32;

template <typename T> __global__ void __launch_bounds__(kPrepThreads) latent_prepare_kernel(const nb_latent_prepare_args p) {
  __shared__ float red[4 * kPrepWarps];
  pdl_enter();
  const int row = blockIdx.x, b = row / p.T, t = row - b * p.T, tid = threadIdx.x;
  const T* a = reinterpret_cast<const T*>(p.a) + (size_t)row * p.lda;
  float mean, inv;
  {
    const T* q = a + p.q_off;
    norm_stats<kPrepWarps>(NB_NORM_RMS, p.q_rank, p.eps, red,
                           [&](auto f) { for (int i = tid; i < p.q_rank; i += kPrepThreads) f(to_f(q[i])); }, mean, inv);
    T* cq = reinterpret_cast<T*>(p.cq) + (size_t)row * p.ldcq;
    for (int i = tid; i < p.q_rank; i += kPrepThreads) cq[i] = from_f<T>(to_f(q[i]) * inv * p.q_norm[i]);
  }
  if (p.kv_off >= 0) {
    const T* kv = a + p.kv_off;
    norm_stats<kPrepWarps>(NB_NORM_RMS, p.rank, p.eps, red + 2 * kPrepWarps,
                           [&](auto f) { for (int i = tid; i < p.rank; i += kPrepThreads) f(to_f(kv[i])); }, mean, inv);
    const int pos = p.pos0 + t;
    T* c = reinterpret_cast<T*>(p.cache) + ((size_t)b * p.ctx + pos) * p.ldc;
    for (int i = tid; i < p.rank; i += kPrepThreads) c[i] = from_f<T>(to_f(kv[i]) * inv * p.kv_norm[i]);
    const float *cs = p.cos2 + (size_t)pos * p.rot, *sn = p.sin2 + (size_t)pos * p.rot;
    for (int d = tid; d < p.rot; d += kPrepThreads)
      c[p.rank + d] = from_f<T>(rotated([&](int i) { return to_f(kv[p.rank + i]); }, cs, sn, d));
  }
}

// Eight bf16 values (four pairs) of a rotated vector; c, s: their entries of the tables.
__device__ __forceinline__ uint4 rotate8(uint4 t, const float* __restrict__ c, const float* __restrict__ s) {
  const float4 c0 = __ldg(reinterpret_cast<const float4*>(c)), c1 = __ldg(reinterpret_cast<const float4*>(c + 4));
  const float4 s0 = __ldg(reinterpret_cast<const float4*>(s)), s1 = __ldg(reinterpret_cast<const float4*>(s + 4));
  const float cs[8] = {c0.x, c0.y, c0.z, c0.w, c1.x, c1.y, c1.z, c1.w}, sn[8] = {s0.x, s0.y, s0.z, s0.w, s1.x, s1.y, s1.z, s1.w};
  const uint32_t u[4] = {t.x, t.y, t.z, t.w};
  uint32_t r[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float x = bf_lo(u[e]), y = bf_hi(u[e]);
    r[e] = pack_bf16(x * cs[2 * e] - y * sn[2 * e], y * cs[2 * e + 1] + x * sn[2 * e + 1]);
  }
  return make_uint4(r[0], r[1], r[2], r[3]);
}

// The same for bf16 rows whose pieces are all multiples of eight: one warp per query latent, one per key/value row, sixteen
// bytes per lane and load, everything of a row in flight at once and kept in registers between the norm's two passes.
constexpr int kPvQ = 8;                // loads per lane: up to 2048 columns

template <int N> __device__ __forceinline__ void norm_row_bf16(const bf16* __restrict__ src, const float* __restrict__ w, float eps, int cols,
                                                               bf16* __restrict__ dst, int lane) {
  uint4 v[N];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = (i * 32 + lane) * 8;
    v[i] = c < cols ? *reinterpret_cast<const uint4*>(src + c) : make_uint4(0u, 0u, 0u, 0u);
  }
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const uint32_t u[4] = {v[i].x, v[i].y, v[i].z, v[i].w};
#pragma unroll
    for (int e = 0; e < 4; ++e) ss += bf_lo(u[e]) * bf_lo(u[e]) + bf_hi(u[e]) * bf_hi(u[e]);
  }
  const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)cols + eps);
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = (i * 32 + lane) * 8;
    if (c < cols) {
      const uint32_t u[4] = {v[i].x, v[i].y, v[i].z, v[i].w};
      const float4 a = __ldg(reinterpret_cast<const float4*>(w + c)), b = __ldg(reinterpret_cast<const float4*>(w + c + 4));
      const float wv[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
      uint32_t r[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) r[e] = pack_bf16(bf_lo(u[e]) * inv * wv[2 * e], bf_hi(u[e]) * inv * wv[2 * e + 1]);
      *reinterpret_cast<uint4*>(dst + c) = make_uint4(r[0], r[1], r[2], r[3]);
    }
  }
}

__global__ void __launch_bounds__(256) latent_prepare_vec_kernel(const nb_latent_prepare_args p, int rows) {
  pdl_enter();
  const int lane = threadIdx.x & 31, unit = blockIdx.x * 8 + (threadIdx.x >> 5);
  const bool is_kv = unit >= rows;
  const int row = is_kv ? unit - rows : unit;
  if (row >= rows || (is_kv && p.kv_off < 0)) return;
  const bf16* a = reinterpret_cast<const bf16*>(p.a) + (size_t)row * p.lda;
  if (!is_kv) {
    bf16* cq = reinterpret_cast<bf16*>(p.cq) + (size_t)row * p.ldcq;
    if (p.q_rank <= 1024) norm_row_bf16<kPvQ / 2>(a + p.q_off, p.q_norm, p.eps, p.q_rank, cq, lane);
    else norm_row_bf16<kPvQ>(a + p.q_off, p.q_norm, p.eps, p.q_rank, cq, lane);
    return;
  }
  const int b = row / p.T, pos = p.pos0 + row - b * p.T;
  bf16* c = reinterpret_cast<bf16*>(p.cache) + ((size_t)b * p.ctx + pos) * p.ldc;
  const bf16* kv = a + p.kv_off;
  if (p.rank <= 512) norm_row_bf16<2>(kv, p.kv_norm, p.eps, p.rank, c, lane);
  else norm_row_bf16<kPvQ>(kv, p.kv_norm, p.eps, p.rank, c, lane);
  const float *cs = p.cos2 + (size_t)pos * p.rot, *sn = p.sin2 + (size_t)pos * p.rot;
  for (int d = lane * 8; d < p.rot; d += 256)
    *reinterpret_cast<uint4*>(c + p.rank + d) = rotate8(*reinterpret_cast<const uint4*>(kv + p.rank + d), cs + d, sn + d);
}

// ---- a portion of a prompt, fp32.  A CTA owns 16 queries of one head and walks the visible keys in chunks of 32 staged
// in shared memory; eight threads share a query (every eighth key for the scores, every eighth value for the sums).
constexpr int kLQ = 16, kLK = 32, kLThreads = 128;

template <int VPT>   // values per thread: vdim <= 8 * VPT
__global__ void __launch_bounds__(kLThreads) latent_attention_f32_kernel(const nb_latent_attention_args p) {
  extern __shared__ __align__(16) float lsm[];
  const int dk = p.dim + p.rot, dkp = dk + 1, vp = p.vdim + 1;
  float* q_s = lsm;                       // [kLQ][dkp]
  float* k_s = q_s + kLQ * dkp;           // [kLK][dkp]
  float* v_s = k_s + kLK * dkp;           // [kLK][vp]
  float* p_s = v_s + kLK * vp;            // [kLQ][kLK + 1]
  const int tid = threadIdx.x, q0 = blockIdx.x * kLQ, h = blockIdx.y, b = blockIdx.z;
  const float* q = reinterpret_cast<const float*>(p.q);
  const float* kv = reinterpret_cast<const float*>(p.kv) + (size_t)b * p.kv_rows * p.ldkv;
  const float* cache = reinterpret_cast<const float*>(p.cache) + (size_t)b * p.ctx * p.ldc;

  for (int i = tid; i < kLQ * dk; i += kLThreads) {
    const int r = i / dk, d = i - r * dk, t = min(q0 + r, p.T - 1);
    const float* qr = q + (size_t)(b * p.T + t) * p.ldq + h * dk;
    float v;
    if (d < p.dim) {
      v = qr[d];
    } else {
      const size_t at = (size_t)(p.pos0 + t) * p.rot;
      v = rotated([&](int j) { return qr[p.dim + j]; }, p.cos2 + at, p.sin2 + at, d - p.dim);
    }
    q_s[r * dkp + d] = v;
  }
  const int qi = tid >> 3, sub = tid & 7;
  const int my_pos = p.pos0 + min(q0 + qi, p.T - 1);
  const int first = p.window > 0 ? max(0, p.pos0 + q0 - p.window + 1) : 0;
  const int last = p.pos0 + min(q0 + kLQ - 1, p.T - 1);
  float m = -INFINITY, l = 0.f, acc[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) acc[i] = 0.f;

  for (int kc = first; kc <= last; kc += kLK) {
    __syncthreads();                      // the chunk before is no longer read
    for (int i = tid; i < kLK * dk; i += kLThreads) {
      const int j = i / dk, d = i - j * dk, pos = kc + j;
      float v = 0.f;
      if (pos <= last)
        v = d < p.dim ? kv[(size_t)(pos - p.kv_pos0) * p.ldkv + h * p.dim + d] : cache[(size_t)pos * p.ldc + p.rank + d - p.dim];
      k_s[j * dkp + d] = v;
    }
    for (int i = tid; i < kLK * p.vdim; i += kLThreads) {
      const int j = i / p.vdim, d = i - j * p.vdim, pos = kc + j;
      v_s[j * vp + d] = pos <= last ? kv[(size_t)(pos - p.kv_pos0) * p.ldkv + p.v_off + h * p.vdim + d] : 0.f;
    }
    __syncthreads();
    float sc[4] = {0.f, 0.f, 0.f, 0.f}, cm = -INFINITY;
    for (int d = 0; d < dk; ++d) {
      const float x = q_s[qi * dkp + d];
#pragma unroll
      for (int i = 0; i < 4; ++i) sc[i] = fmaf(x, k_s[(sub + 8 * i) * dkp + d], sc[i]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int pos = kc + sub + 8 * i;
      const bool seen = pos <= my_pos && (p.window <= 0 || my_pos - pos < p.window);
      sc[i] = seen ? sc[i] * p.scale : -INFINITY;
      cm = fmaxf(cm, sc[i]);
    }
#pragma unroll
    for (int o = 1; o < 8; o <<= 1) cm = fmaxf(cm, __shfl_xor_sync(0xffffffffu, cm, o));
    const float m_new = fmaxf(m, cm), base = m_new == -INFINITY ? 0.f : m_new;   // nothing seen so far: all weights are 0
    const float corr = expf(m - base);
    float ps = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float e = expf(sc[i] - base);
      p_s[qi * (kLK + 1) + sub + 8 * i] = e;
      ps += e;
    }
#pragma unroll
    for (int o = 1; o < 8; o <<= 1) ps += __shfl_xor_sync(0xffffffffu, ps, o);
    l = l * corr + ps;
    m = m_new;
#pragma unroll
    for (int i = 0; i < VPT; ++i) acc[i] *= corr;
    __syncwarp();                         // the eight threads of a query are lanes of one warp
    for (int j = 0; j < kLK; ++j) {
      const float w = p_s[qi * (kLK + 1) + j];
#pragma unroll
      for (int i = 0; i < VPT; ++i)
        if (sub + 8 * i < p.vdim) acc[i] = fmaf(w, v_s[j * vp + sub + 8 * i], acc[i]);
    }
  }
  if (q0 + qi < p.T) {
    const size_t row = (size_t)b * p.T + q0 + qi;
    const float g = (p.gate ? sigmoid_f(reinterpret_cast<const float*>(p.gate)[row * p.ldg + h]) : 1.f) / l;
    float* o = reinterpret_cast<float*>(p.out) + row * p.ldo + h * p.vdim;
#pragma unroll
    for (int i = 0; i < VPT; ++i)
      if (sub + 8 * i < p.vdim) o[sub + 8 * i] = acc[i] * g;
  }
}

// ---- a portion of a prompt, bf16 operands.  A CTA of four warps owns 64 queries of one head (16 per warp) and walks the
// visible keys in tiles of 64; the next tile's keys and values are copied while this one is multiplied (two stages).
// Scores and the running softmax are fp32; the softmax weights enter the second product as two bf16 terms, so that they
// are not rounded to eight bits.
constexpr int kTQ = 64, kTK = 64, kTThreads = 128;

template <int VD>
__global__ void __launch_bounds__(kTThreads) latent_attention_bf16_kernel(const nb_latent_attention_args p, int dk16, int vec, int qvec) {
  extern __shared__ __align__(16) bf16 tsm[];
  const int dk = p.dim + p.rot, dkp = dk16 + 8;
  constexpr int vp = VD + 8;
  bf16* q_s = tsm;                              // [kTQ][dkp]
  bf16* k_s = q_s + kTQ * dkp;                  // [2][kTK][dkp]
  bf16* v_s = k_s + 2 * kTK * dkp;              // [2][kTK][vp]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int q0 = (gridDim.x - 1 - blockIdx.x) * kTQ, h = blockIdx.y, b = blockIdx.z;
  const bf16* q = reinterpret_cast<const bf16*>(p.q);
  const bf16* kv = reinterpret_cast<const bf16*>(p.kv) + (size_t)b * p.kv_rows * p.ldkv;
  const bf16* cache = reinterpret_cast<const bf16*>(p.cache) + (size_t)b * p.ctx * p.ldc;
  const int first = p.window > 0 ? max(0, p.pos0 + q0 - p.window + 1) : 0;
  const int last = p.pos0 + min(q0 + kTQ - 1, p.T - 1);
  const int tiles = (last - first) / kTK + 1;

  // columns past dk (keys, queries) and past vdim (values) stay zero
  for (int i = tid; i < 3 * kTK * (dkp - dk); i += kTThreads) {
    const int r = i / (dkp - dk);
    q_s[r * dkp + dk + i - r * (dkp - dk)] = from_f<bf16>(0.f);
  }
  for (int i = tid; i < 2 * kTK * (vp - p.vdim); i += kTThreads) {
    const int r = i / (vp - p.vdim);
    v_s[r * vp + p.vdim + i - r * (vp - p.vdim)] = from_f<bf16>(0.f);
  }

  auto copy_tile = [&](int tile, int st) {
    const int k0 = first + tile * kTK;
    bf16* kd = k_s + st * kTK * dkp;
    bf16* vd = v_s + st * kTK * vp;
    if (vec) {
      // eight threads per row, 16 bytes each: 128 consecutive bytes of one piece at a time
      const int c8 = (tid & 7) * 8;
#pragma unroll
      for (int jr = 0; jr < kTK; jr += kTThreads / 8) {
        const int j = jr + (tid >> 3), pos = k0 + j;
        bf16 *kr = kd + j * dkp, *vr = vd + j * vp;
        if (pos <= last) {
          const bf16* row = kv + (size_t)(pos - p.kv_pos0) * p.ldkv;
          const bf16* cr = cache + (size_t)pos * p.ldc + p.rank;
          for (int c = c8; c < p.dim; c += 64) cp16(kr + c, row + h * p.dim + c);
          for (int c = c8; c < p.rot; c += 64) cp16(kr + p.dim + c, cr + c);
          for (int c = c8; c < p.vdim; c += 64) cp16(vr + c, row + p.v_off + h * p.vdim + c);
        } else {
          for (int c = c8; c < dk; c += 64) *reinterpret_cast<uint4*>(kr + c) = make_uint4(0u, 0u, 0u, 0u);
          for (int c = c8; c < p.vdim; c += 64) *reinterpret_cast<uint4*>(vr + c) = make_uint4(0u, 0u, 0u, 0u);
        }
      }
    } else {
      const int n = dk + p.vdim;
      for (int i = tid; i < kTK * n; i += kTThreads) {
        const int j = i / n, c = i - j * n, pos = k0 + j;
        bf16 v = from_f<bf16>(0.f);
        if (pos <= last) {
          const bf16* row = kv + (size_t)(pos - p.kv_pos0) * p.ldkv;
          v = c < p.dim ? row[h * p.dim + c] : c < dk ? cache[(size_t)pos * p.ldc + p.rank + c - p.dim] : row[p.v_off + h * p.vdim + c - dk];
        }
        if (c < dk) kd[j * dkp + c] = v;
        else vd[j * vp + c - dk] = v;
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (qvec) {                                   // travels with the first tile; the rotated part through registers
    const int c8 = (tid & 7) * 8;
#pragma unroll
    for (int r0 = 0; r0 < kTQ; r0 += kTThreads / 8) {
      const int r = r0 + (tid >> 3), t = min(q0 + r, p.T - 1);
      const bf16* qr = q + (size_t)(b * p.T + t) * p.ldq + h * dk;
      for (int c = c8; c < p.dim; c += 64) cp16(q_s + r * dkp + c, qr + c);
    }
  }
  copy_tile(0, 0);
  if (qvec) {
    const int c8 = (tid & 7) * 8;
#pragma unroll
    for (int r0 = 0; r0 < kTQ; r0 += kTThreads / 8) {
      const int r = r0 + (tid >> 3), t = min(q0 + r, p.T - 1);
      const bf16* qr = q + (size_t)(b * p.T + t) * p.ldq + h * dk + p.dim;
      const float *cs = p.cos2 + (size_t)(p.pos0 + t) * p.rot, *sn = p.sin2 + (size_t)(p.pos0 + t) * p.rot;
      for (int c = c8; c < p.rot; c += 64)
        *reinterpret_cast<uint4*>(q_s + r * dkp + p.dim + c) = rotate8(*reinterpret_cast<const uint4*>(qr + c), cs + c, sn + c);
    }
  } else {
    for (int i = tid; i < kTQ * dk; i += kTThreads) {
      const int r = i / dk, d = i - r * dk, t = min(q0 + r, p.T - 1);
      const bf16* qr = q + (size_t)(b * p.T + t) * p.ldq + h * dk;
      bf16 v;
      if (d < p.dim) {
        v = qr[d];
      } else {
        const size_t at = (size_t)(p.pos0 + t) * p.rot;
        v = from_f<bf16>(rotated([&](int j) { return to_f(qr[p.dim + j]); }, p.cos2 + at, p.sin2 + at, d - p.dim));
      }
      q_s[r * dkp + d] = v;
    }
  }

  // this lane's two rows of the warp's 16 queries: lane / 4 and lane / 4 + 8
  const int rowa = warp * 16 + (lane >> 2);
  const int pos_a = p.pos0 + min(q0 + rowa, p.T - 1), pos_b = p.pos0 + min(q0 + rowa + 8, p.T - 1);
  const int wlo = p.pos0 + min(q0 + warp * 16, p.T - 1), whi = p.pos0 + min(q0 + warp * 16 + 15, p.T - 1);   // of the warp's queries
  const float sl2 = p.scale * 1.4426950408889634f;     // softmax in base 2
  float o[VD / 8][4];
#pragma unroll
  for (int i = 0; i < VD / 8; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) o[i][j] = 0.f;
  float ma = -INFINITY, mb = -INFINITY, la = 0.f, lb = 0.f;

  for (int tile = 0; tile < tiles; ++tile) {
    const int st = tile & 1, k0 = first + tile * kTK;
    if (tile + 1 < tiles) {
      copy_tile(tile + 1, st ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const bf16* kt = k_s + st * kTK * dkp;
    const bf16* vt = v_s + st * kTK * vp;
    float s[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) s[i][j] = 0.f;
#pragma unroll 4
    for (int kk = 0; kk < dk16; kk += 16) {
      uint32_t a[4];
      ldsm_x4(a, q_s + (warp * 16 + (lane & 15)) * dkp + kk + (lane >> 4) * 8);
#pragma unroll
      for (int n = 0; n < 4; ++n) {                    // 16 keys per load
        uint32_t bb[4];
        ldsm_x4(bb, kt + (n * 16 + (lane & 7) + ((lane >> 4) << 3)) * dkp + kk + ((lane >> 3) & 1) * 8);
        mma_bf16(s[2 * n], a, bb[0], bb[1]);
        mma_bf16(s[2 * n + 1], a, bb[2], bb[3]);
      }
    }
    // a tile that every query of the warp sees whole needs no mask
    const bool whole = k0 + kTK - 1 <= wlo && (p.window <= 0 || whi - k0 < p.window);
    if (!whole) {
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int pos = k0 + n * 8 + (lane & 3) * 2 + (j & 1), me = j < 2 ? pos_a : pos_b;
          if (!(pos <= me && (p.window <= 0 || me - pos < p.window))) s[n][j] = -INFINITY;
        }
    }
    float na = ma, nb_ = mb;
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      na = fmaxf(na, fmaxf(s[n][0], s[n][1]));
      nb_ = fmaxf(nb_, fmaxf(s[n][2], s[n][3]));
    }
#pragma unroll
    for (int x = 1; x < 4; x <<= 1) {
      na = fmaxf(na, __shfl_xor_sync(0xffffffffu, na, x));
      nb_ = fmaxf(nb_, __shfl_xor_sync(0xffffffffu, nb_, x));
    }
    // ma, mb: largest score so far, before the scale (which is positive)
    const float ba = na == -INFINITY ? 0.f : na * sl2, bb_ = nb_ == -INFINITY ? 0.f : nb_ * sl2;   // nothing seen yet: all weights are 0
    const float ca = ex2(fmaf(ma, sl2, -ba)), cb = ex2(fmaf(mb, sl2, -bb_));
    ma = na; mb = nb_;
    la *= ca; lb *= cb;
#pragma unroll
    for (int i = 0; i < VD / 8; ++i) { o[i][0] *= ca; o[i][1] *= ca; o[i][2] *= cb; o[i][3] *= cb; }
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      s[n][0] = ex2(fmaf(s[n][0], sl2, -ba)); s[n][1] = ex2(fmaf(s[n][1], sl2, -ba));
      s[n][2] = ex2(fmaf(s[n][2], sl2, -bb_)); s[n][3] = ex2(fmaf(s[n][3], sl2, -bb_));
      la += s[n][0] + s[n][1];
      lb += s[n][2] + s[n][3];
    }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {                   // 16 keys per step
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {                    // registers of the A fragment: (row a, keys 0-7), (row b, ..), (row a, keys 8-15), (row b, ..)
        const float x = s[2 * kk + (j >> 1)][(j & 1) * 2], y = s[2 * kk + (j >> 1)][(j & 1) * 2 + 1];
        split_bf16(x, y, hi[j], lo[j]);
      }
#pragma unroll
      for (int n = 0; n < VD / 16; n += 2) {           // four independent products before an accumulator comes again
        uint32_t bb[2][4];
        ldsm_x4_t(bb[0], vt + (kk * 16 + (lane & 15)) * vp + n * 16 + (lane >> 4) * 8);
        ldsm_x4_t(bb[1], vt + (kk * 16 + (lane & 15)) * vp + n * 16 + 16 + (lane >> 4) * 8);
#pragma unroll
        for (int term = 0; term < 2; ++term)
#pragma unroll
          for (int y = 0; y < 2; ++y)
#pragma unroll
            for (int x = 0; x < 2; ++x) mma_bf16(o[2 * (n + y) + x], term ? lo : hi, bb[y][2 * x], bb[y][2 * x + 1]);
      }
    }
    __syncthreads();                                   // before the stage is filled again
  }
#pragma unroll
  for (int x = 1; x < 4; x <<= 1) {
    la += __shfl_xor_sync(0xffffffffu, la, x);
    lb += __shfl_xor_sync(0xffffffffu, lb, x);
  }
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int r = q0 + rowa + 8 * half;
    if (r >= p.T) continue;
    const size_t row = (size_t)b * p.T + r;
    const float g = (p.gate ? sigmoid_f(to_f(reinterpret_cast<const bf16*>(p.gate)[row * p.ldg + h])) : 1.f) / (half ? lb : la);
    bf16* out = reinterpret_cast<bf16*>(p.out) + row * p.ldo + h * p.vdim;
#pragma unroll
    for (int i = 0; i < VD / 8; ++i) {
      const int d = i * 8 + (lane & 3) * 2;
      if (vec) {
        if (d < p.vdim) *reinterpret_cast<uint32_t*>(out + d) = pack_bf16(o[i][2 * half] * g, o[i][2 * half + 1] * g);
      } else {
        if (d < p.vdim) out[d] = from_f<bf16>(o[i][2 * half] * g);
        if (d + 1 < p.vdim) out[d + 1] = from_f<bf16>(o[i][2 * half + 1] * g);
      }
    }
  }
}

// ---- one position per sequence.  grid (H, B, S) in clusters of S CTAs along z.  The CTAs of a head share its work three
// times over: slices of the latent for q' = W_uk^T q, contiguous ranges of the window's keys for the softmax and the
// weighted latent, slices of the values for W_uv; the slices travel through distributed shared memory.  A CTA's cached rows
// are staged in shared memory (`stage` of them at a time, with a running maximum and sum if there are more) and serve as keys
// and as values from there.  Everything that does not depend on the launch before — the rows of earlier positions, the
// weights — is requested ahead of the dependency wait.
constexpr int kLdThreads = 256, kLdWarps = kLdThreads / 32;
constexpr int kLdCols = 2;             // groups of four columns per thread: rank <= 4 * 256 * 2
constexpr int kLdPre = 16;             // W_uk words a thread may hold ahead of the wait

__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

template <typename T> __device__ __forceinline__ float dot16(const void* row16, const float* __restrict__ q);
template <> __device__ __forceinline__ float dot16<bf16>(const void* r, const float* __restrict__ q) {      // eight bf16
  const uint4 t = *reinterpret_cast<const uint4*>(r);
  const float4 a = *reinterpret_cast<const float4*>(q), b = *reinterpret_cast<const float4*>(q + 4);
  return bf_lo(t.x) * a.x + bf_hi(t.x) * a.y + bf_lo(t.y) * a.z + bf_hi(t.y) * a.w + bf_lo(t.z) * b.x + bf_hi(t.z) * b.y + bf_lo(t.w) * b.z +
         bf_hi(t.w) * b.w;
}
template <> __device__ __forceinline__ float dot16<float>(const void* r, const float* __restrict__ q) {     // four fp32
  const float4 t = *reinterpret_cast<const float4*>(r), a = *reinterpret_cast<const float4*>(q);
  return t.x * a.x + t.y * a.y + t.z * a.z + t.w * a.w;
}
__device__ __forceinline__ float4 quad_at(const bf16* r) {
  const uint2 t = *reinterpret_cast<const uint2*>(r);
  return make_float4(bf_lo(t.x), bf_hi(t.x), bf_lo(t.y), bf_hi(t.y));
}
__device__ __forceinline__ float4 quad_at(const float* r) { return *reinterpret_cast<const float4*>(r); }

// Sixteen bytes of a staged row times the matching part of the query.
__device__ __forceinline__ float dot_piece(const bf16* r, const float (&q)[8]) {
  const uint4 t = *reinterpret_cast<const uint4*>(r);
  return (bf_lo(t.x) * q[0] + bf_hi(t.x) * q[1]) + (bf_lo(t.y) * q[2] + bf_hi(t.y) * q[3]) + (bf_lo(t.z) * q[4] + bf_hi(t.z) * q[5]) +
         (bf_lo(t.w) * q[6] + bf_hi(t.w) * q[7]);
}
__device__ __forceinline__ float dot_piece(const float* r, const float (&q)[4]) {
  const float4 t = *reinterpret_cast<const float4*>(r);
  return (t.x * q[0] + t.y * q[1]) + (t.z * q[2] + t.w * q[3]);
}

template <typename T>
__global__ void __launch_bounds__(kLdThreads, 2) latent_decode_kernel(const nb_latent_decode_args p, int stage) {
  extern __shared__ __align__(16) float dsm[];
  __shared__ float red[kLdWarps], red2[kLdWarps], red3[kLdWarps];
  cg::cluster_group cluster = cg::this_cluster();
  const int S = (int)cluster.num_blocks(), rank_id = (int)cluster.block_rank();
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int rd = p.rank + p.rot, dk = p.dim + p.rot, rdp = (rd + 7) & ~7, ldr = rdp;
  float* qa = dsm;                     // [rdp] q' and the rotated query part: what the cached rows are multiplied with
  float* ol = qa + rdp;                // [rdp] merged latent
  float* qn = ol + rdp;                // [dk] this head's query
  float* cs = qn + ((dk + 7) & ~7);    // [rot] the position's rotary entries
  float* sn = cs + ((p.rot + 7) & ~7);
  float* part = sn + ((p.rot + 7) & ~7);   // [kLdThreads * 4] partial sums
  const int pairs = (p.rank + 1) / 2, pper = (pairs + S - 1) / S, slot = (2 * pper + 2 + 3) & ~3;
  float* xch = part + 4 * kLdThreads;  // [S][slot] what the CTAs send: their part of this CTA's slice, maximum, sum
  float* sc = xch + S * slot;          // [stage] scores, then weights, of the staged keys
  T* rows = reinterpret_cast<T*>(sc + ((stage + 3) & ~3));   // [stage][ldr]

  // The position was written at the end of the step before, the rows below it in earlier steps or the prompt.
  const long long pos = *p.pos;
  if (pos < 0 || pos >= p.ctx) return; // the same for every CTA
  const int n = p.window > 0 ? min((int)pos + 1, p.window) : (int)pos + 1, first = (int)pos + 1 - n;
  const int per = (n + S - 1) / S, k0 = first + rank_id * per, cnt = max(0, min(first + n, k0 + per) - k0);
  T* cache = reinterpret_cast<T*>(p.cache) + (size_t)b * p.ctx * p.ldc;
  constexpr int kPiece = 16 / sizeof(T);
  const int pieces = rdp / kPiece;
  auto request = [&](int base, int m) {       // rows k0 + base .. of earlier positions
    for (int j = warp; j < m; j += kLdWarps) {
      if (k0 + base + j == (int)pos) continue;
      const T* src = cache + (size_t)(k0 + base + j) * p.ldc;
      T* dst = rows + (size_t)j * ldr;
      for (int c = lane; c < pieces; c += 32) cp16(dst + c * kPiece, src + c * kPiece);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  request(0, min(stage, cnt));

  // W_uk: this CTA's slice of columns (pairs), the d range split over groups of threads
  const int p0 = rank_id * pper, pn = max(0, min(pairs, p0 + pper) - p0);
  const bf16* uk = reinterpret_cast<const bf16*>(p.uk) + (size_t)h * p.dim * p.ldu;
  const int cols0 = min(pn, kLdThreads), groups0 = cols0 ? kLdThreads / cols0 : 1, g0 = cols0 ? tid / cols0 : 0, c0 = cols0 ? tid - g0 * cols0 : 0;
  const bool pre = pn > 0 && pn <= kLdThreads && (p.dim + groups0 - 1) / groups0 <= kLdPre;
  uint32_t wreg[kLdPre];
#pragma unroll
  for (int i = 0; i < kLdPre; ++i) {
    const int d = g0 + i * groups0;
    wreg[i] = (pre && g0 < groups0 && d < p.dim) ? __ldg(reinterpret_cast<const uint32_t*>(uk + (size_t)d * p.ldu + 2 * (p0 + c0))) : 0u;
  }
  const int vper = (p.vdim + S - 1) / S, v0 = rank_id * vper, v1 = min(p.vdim, v0 + vper);
  const bf16* uv = reinterpret_cast<const bf16*>(p.uv) + (size_t)h * p.vdim * p.ldu;
  for (int i = tid; i < (v1 - v0) * ((p.rank + 63) / 64); i += kLdThreads) {
    const int v = i / ((p.rank + 63) / 64), c = i - v * ((p.rank + 63) / 64);
    prefetch_l2(uv + (size_t)(v0 + v) * p.ldu + c * 64);
  }
  // the position's rotary entries and the norm's weights
  const float* ct = p.cos2 + (size_t)pos * p.rot;
  const float* stb = p.sin2 + (size_t)pos * p.rot;
  const float c_pre = tid < p.rot ? ct[tid] : 0.f, s_pre = tid < p.rot ? stb[tid] : 0.f;
  const int mine = (int)pos - k0;      // this position's place among this CTA's keys, if 0 <= mine < cnt
  const bool holds = mine >= 0 && mine < cnt;
  constexpr int kKv = 4 * kLdCols;     // elements of the position's latent per thread
  float kvw[kKv], kvv[kKv];
  if (p.kv_off >= 0 && holds) {
#pragma unroll
    for (int u = 0; u < kKv; ++u) kvw[u] = tid + u * kLdThreads < p.rank ? p.kv_norm[tid + u * kLdThreads] : 0.f;
  }
  for (int j = stage + warp; j < cnt; j += kLdWarps)     // rows that are staged later: on their way to L2
    for (int c = lane * (64 / (int)sizeof(T)) * 2; c < rd; c += 32 * (64 / (int)sizeof(T)) * 2)
      prefetch_l2(cache + (size_t)(k0 + j) * p.ldc + c);
  cluster.barrier_arrive();

  pdl_enter();
  if (tid < p.rot) { cs[tid] = c_pre; sn[tid] = s_pre; }
  for (int i = tid + kLdThreads; i < p.rot; i += kLdThreads) { cs[i] = ct[i]; sn[i] = stb[i]; }
  for (int i = tid; i < dk; i += kLdThreads) qn[i] = p.q[(size_t)b * p.ldq + h * dk + i];
  const float gate = p.a[(size_t)b * p.lda + p.g_off + h];
  for (int i = rd + tid; i < rdp; i += kLdThreads) qa[i] = 0.f;
  // this position's row, into its staged place: from the projection (and then written to the cache by one CTA) or from
  // the cache.  With more keys than are staged at a time it waits in its registers for its turn.
  float inv = 0.f;
  const float* kv = p.a + (size_t)b * p.lda + max(p.kv_off, 0);
  if (p.kv_off >= 0 && holds) {        // block-uniform
    float ss = 0.f;
#pragma unroll
    for (int u = 0; u < kKv; ++u) {
      kvv[u] = tid + u * kLdThreads < p.rank ? kv[tid + u * kLdThreads] : 0.f;
      ss += kvv[u] * kvv[u];
    }
    inv = 1.0f / sqrtf(block_sum<kLdWarps>(ss, red) / (float)p.rank + p.eps);
  } else {
    __syncthreads();                   // the query and the rotary entries
  }
  auto put_row = [&](T* dst) {         // dst: the staged row
    T* crow = cache + (size_t)pos * p.ldc;
    if (p.kv_off >= 0) {
#pragma unroll
      for (int u = 0; u < kKv; ++u) {
        const int i = tid + u * kLdThreads;
        if (i < p.rank) {
          const T v = from_f<T>(kvv[u] * inv * kvw[u]);
          dst[i] = v;
          if (h == 0) crow[i] = v;
        }
      }
      for (int d = tid; d < p.rot; d += kLdThreads) {
        const T v = from_f<T>(rotated([&](int j) { return kv[p.rank + j]; }, cs, sn, d));
        dst[p.rank + d] = v;
        if (h == 0) crow[p.rank + d] = v;
      }
    } else {
      for (int i = tid; i < rd; i += kLdThreads) dst[i] = crow[i];
    }
    for (int i = rd + tid; i < rdp; i += kLdThreads) dst[i] = from_f<T>(0.f);
  };
  if (mine >= 0 && mine < min(stage, cnt)) put_row(rows + (size_t)mine * ldr);
  for (int d = tid; d < p.rot; d += kLdThreads) qa[p.rank + d] = rotated([&](int j) { return qn[p.dim + j]; }, cs, sn, d);

  // q'[j] = sum_d W_uk[h][d][j] q[d]
  for (int base = 0; base < pn; base += kLdThreads) {
    const int cols = min(pn - base, kLdThreads), groups = kLdThreads / cols, gi = tid / cols, c = tid - gi * cols;
    float x = 0.f, y = 0.f;
    if (pre) {
#pragma unroll
      for (int i = 0; i < kLdPre; ++i) {
        const int d = g0 + i * groups0;
        if (d < p.dim) { x = fmaf(bf_lo(wreg[i]), qn[d], x); y = fmaf(bf_hi(wreg[i]), qn[d], y); }
      }
    } else if (gi < groups) {
      const int j = 2 * (p0 + base + c);
#pragma unroll 8
      for (int d = gi; d < p.dim; d += groups) {
        const uint32_t w = *reinterpret_cast<const uint32_t*>(uk + (size_t)d * p.ldu + j);
        x = fmaf(bf_lo(w), qn[d], x);
        y = fmaf(bf_hi(w), qn[d], y);
      }
    }
    part[2 * tid] = x; part[2 * tid + 1] = y;
    if (base == 0) cluster.barrier_wait();     // every CTA of the cluster runs: its shared memory may be written from here on
    __syncthreads();
    for (int i = tid; i < 2 * cols; i += kLdThreads) {
      float v = 0.f;
      for (int g = 0; g < groups; ++g) v += part[2 * g * cols + i];
      const int j = 2 * (p0 + base) + i;
      if (j < p.rank)
        for (int r = 0; r < S; ++r) cluster.map_shared_rank(qa, r)[j] = v;
    }
    __syncthreads();
  }
  if (pn == 0) cluster.barrier_wait();
  cluster.sync();

  // softmax and weighted latent over the staged rows.  Scores: a warp takes four
  // keys at a time, a lane holds its part of the query in registers (shared-memory reads of the query would cost more than
  // those of the rows).  Latent: a
  // thread owns four columns (or kLdCols times four); with few columns the keys are split over `groups` of threads.
  const int quads = (p.rank + 3) / 4;
  const int wcols = min(quads, kLdThreads), groups = quads <= kLdThreads ? kLdThreads / wcols : 1, gi = tid / wcols, wc = tid - gi * wcols;
  float m = -FLT_MAX, l = 0.f;
  float4 acc[kLdCols];
#pragma unroll
  for (int u = 0; u < kLdCols; ++u) acc[u] = make_float4(0.f, 0.f, 0.f, 0.f);
  constexpr int kQp = sizeof(T) == 2 ? 3 : 5;
  float qreg[kQp][kPiece];
#pragma unroll
  for (int x = 0; x < kQp; ++x)
#pragma unroll
    for (int e = 0; e < kPiece; e += 4) {
      const int c = x * 32 + lane;
      const float4 v = c < pieces ? *reinterpret_cast<const float4*>(qa + c * kPiece + e) : make_float4(0.f, 0.f, 0.f, 0.f);
      qreg[x][e] = v.x; qreg[x][e + 1] = v.y; qreg[x][e + 2] = v.z; qreg[x][e + 3] = v.w;
    }
  for (int base = 0; base < cnt; base += stage) {
    const int nk = min(stage, cnt - base);
    if (base > 0) {
      __syncthreads();                 // the rows and weights before are no longer read
      request(base, nk);
    }
    if (base > 0 && mine >= base && mine < base + nk) put_row(rows + (size_t)(mine - base) * ldr);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    float mx = -FLT_MAX;
    for (int j0 = warp * 4; j0 < nk; j0 += kLdWarps * 4) {
      float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int x = 0; x < kQp; ++x) {
        const int c = x * 32 + lane;
        if (c < pieces) {
#pragma unroll
          for (int k = 0; k < 4; ++k) s[k] += dot_piece(rows + (size_t)min(j0 + k, nk - 1) * ldr + c * kPiece, qreg[x]);
        }
      }
      for (int c = kQp * 32 + lane; c < pieces; c += 32)       // wider rows than the registers hold
#pragma unroll
        for (int k = 0; k < 4; ++k) s[k] += dot16<T>(rows + (size_t)min(j0 + k, nk - 1) * ldr + c * kPiece, qa + c * kPiece);
      // four sums over the warp: lanes keep one key each from the second halving on
      const bool hi16 = lane & 16, hi8 = lane & 8;
      float a = hi16 ? s[2] : s[0], b2 = hi16 ? s[3] : s[1];
      a += __shfl_xor_sync(0xffffffffu, hi16 ? s[0] : s[2], 16);
      b2 += __shfl_xor_sync(0xffffffffu, hi16 ? s[1] : s[3], 16);
      float t = hi8 ? b2 : a;
      t += __shfl_xor_sync(0xffffffffu, hi8 ? a : b2, 8);
#pragma unroll
      for (int x = 4; x > 0; x >>= 1) t += __shfl_xor_sync(0xffffffffu, t, x);
      t *= p.scale;
      const int j = j0 + (hi16 ? 2 : 0) + (hi8 ? 1 : 0);
      if (j < nk) {
        if ((lane & 7) == 0) sc[j] = t;
        mx = fmaxf(mx, t);
      }
    }
    mx = warp_max(mx);
    if (lane == 0) red2[warp] = mx;
    __syncthreads();
    float m_new = m;
#pragma unroll
    for (int i = 0; i < kLdWarps; ++i) m_new = fmaxf(m_new, red2[i]);
    const float corr = expf(m - m_new);
    m = m_new;
    float sum = 0.f;
    for (int j = tid; j < nk; j += kLdThreads) {
      const float e = expf(sc[j] - m);
      sc[j] = e;
      sum += e;
    }
    l = l * corr + block_sum<kLdWarps>(sum, red3);   // its barrier also publishes the weights
#pragma unroll
    for (int u = 0; u < kLdCols; ++u) {
      acc[u].x *= corr; acc[u].y *= corr; acc[u].z *= corr; acc[u].w *= corr;
      const int c = wc + u * kLdThreads;
      if (gi < groups && c < quads) {
#pragma unroll 8
        for (int j = gi; j < nk; j += groups) {
          const float w = sc[j];
          const float4 t = quad_at(rows + (size_t)j * ldr + 4 * c);   // columns past the latent: never sent
          acc[u].x = fmaf(w, t.x, acc[u].x);
          acc[u].y = fmaf(w, t.y, acc[u].y);
          acc[u].z = fmaf(w, t.z, acc[u].z);
          acc[u].w = fmaf(w, t.w, acc[u].w);
        }
      }
    }
  }
  // every CTA sends the parts of its weighted latent to the CTAs that merge them: slice r (2 * pper columns) to CTA r
#pragma unroll
  for (int u = 0; u < kLdCols; ++u) {
    if (u * kLdThreads < quads) {      // block-uniform
      reinterpret_cast<float4*>(part)[tid] = acc[u];
      __syncthreads();
      const int cols = min(4 * kLdThreads, p.rank - 4 * u * kLdThreads);
      for (int i = tid; i < cols; i += kLdThreads) {
        float v = 0.f;
        for (int g = 0; g < groups; ++g) v += part[4 * g * wcols + i];
        const int col = 4 * u * kLdThreads + i, to = col / (2 * pper);
        cluster.map_shared_rank(xch, to)[rank_id * slot + col - to * 2 * pper] = v;
      }
      __syncthreads();
    }
  }
  if (tid < S) {
    float* x = cluster.map_shared_rank(xch, tid) + rank_id * slot + 2 * pper;
    x[0] = m;
    x[1] = l;
  }
  // rows of W_uv for the last product, two per warp, requested ahead of the exchange
  constexpr int kUvPre = 4;
  const bool upre = p.rank <= 512 && v1 - v0 <= 2 * kLdWarps;
  uint4 uvr[kUvPre];
#pragma unroll
  for (int i = 0; i < kUvPre; ++i) {
    const int v = v0 + warp + (i >> 1) * kLdWarps, c = (i & 1) * 256 + lane * 8;
    uvr[i] = (upre && v < v1 && c < p.rank) ? __ldg(reinterpret_cast<const uint4*>(uv + (size_t)v * p.ldu + c)) : make_uint4(0u, 0u, 0u, 0u);
  }
  cluster.sync();
  // this CTA's slice of the merged latent, to everyone
  {
    float m_all = -FLT_MAX, den = 0.f, wr[8];
#pragma unroll
    for (int r = 0; r < 8; ++r)
      if (r < S) m_all = fmaxf(m_all, xch[r * slot + 2 * pper]);
#pragma unroll
    for (int r = 0; r < 8; ++r) {      // a CTA without keys has maximum -FLT_MAX and sum 0
      wr[r] = 0.f;
      if (r < S) {
        wr[r] = expf(xch[r * slot + 2 * pper] - m_all);
        den += wr[r] * xch[r * slot + 2 * pper + 1];
      }
    }
    for (int i = tid; i < min(2 * pn, p.rank - 2 * p0); i += kLdThreads) {
      float num = 0.f;
#pragma unroll
      for (int r = 0; r < 8; ++r)
        if (r < S) num += wr[r] * xch[r * slot + i];
      const float v = num / den;
      for (int r = 0; r < S; ++r) cluster.map_shared_rank(ol, r)[2 * p0 + i] = v;
    }
  }
  for (int i = p.rank + tid; i < ((p.rank + 7) & ~7); i += kLdThreads) ol[i] = 0.f;   // W_uv is read in eights
  cluster.sync();                      // also: nobody reads another CTA's shared memory after this
  const float g = sigmoid_f(gate);
  if (upre) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int v = v0 + warp + r * kLdWarps;
      if (v < v1) {
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int c = i * 256 + lane * 8;
          if (c < p.rank) s += dot16<bf16>(&uvr[2 * r + i], ol + c);
        }
        s = warp_sum(s);
        if (lane == 0) p.out[(size_t)b * p.ldo + h * p.vdim + v] = s * g;
      }
    }
  } else {
    for (int v = v0 + warp; v < v1; v += kLdWarps) {
      const bf16* wv = uv + (size_t)v * p.ldu;
      float s = 0.f;
      for (int i = lane * 8; i < p.rank; i += 256) s += dot16<bf16>(wv + i, ol + i);
      s = warp_sum(s);
      if (lane == 0) p.out[(size_t)b * p.ldo + h * p.vdim + v] = s * g;
    }
  }
}

constexpr size_t kLatentMaxSmem = 200 * 1024, kLatentHalfSmem = 110 * 1024;

template <int VPT> static int launch_latent_f32(const nb_latent_attention_args& a, cudaStream_t st) {
  const int dk = a.dim + a.rot;
  const size_t smem = ((size_t)(kLQ + kLK) * (dk + 1) + (size_t)kLK * (a.vdim + 1) + kLQ * (kLK + 1)) * 4;
  if (smem > kLatentMaxSmem) return NB_ERR_SHAPE;
  static bool done[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!done[dev & 63]) {
    if (cudaError_t e = cudaFuncSetAttribute(latent_attention_f32_kernel<VPT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLatentMaxSmem))
      return record_cuda_error(e);
    done[dev & 63] = true;
  }
  latent_attention_f32_kernel<VPT><<<dim3((a.T + kLQ - 1) / kLQ, a.H, a.B), kLThreads, smem, st>>>(a);
  return check_launch();
}

template <int VD> static int launch_latent_bf16(const nb_latent_attention_args& a, cudaStream_t st) {
  const int dk16 = (a.dim + a.rot + 15) & ~15;
  const size_t smem = ((size_t)3 * kTK * (dk16 + 8) + (size_t)2 * kTK * (VD + 8)) * 2;
  if (smem > kLatentMaxSmem) return NB_ERR_SHAPE;
  static bool done[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!done[dev & 63]) {
    if (cudaError_t e = cudaFuncSetAttribute(latent_attention_bf16_kernel<VD>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLatentMaxSmem))
      return record_cuda_error(e);
    done[dev & 63] = true;
  }
  // 16-byte copies need every piece of a row to start and end on 16 bytes
  const int vec = a.dim % 8 == 0 && a.rot % 8 == 0 && a.vdim % 8 == 0 && a.rank % 8 == 0 && a.ldkv % 8 == 0 && a.ldc % 8 == 0 &&
                  a.v_off % 8 == 0 && a.ldo % 2 == 0 && (uintptr_t)a.kv % 16 == 0 && (uintptr_t)a.cache % 16 == 0 && (uintptr_t)a.out % 4 == 0;
  const int qvec = a.dim % 8 == 0 && a.rot % 8 == 0 && a.ldq % 8 == 0 && (uintptr_t)a.q % 16 == 0 && (uintptr_t)a.cos2 % 16 == 0 &&
                   (uintptr_t)a.sin2 % 16 == 0;
  latent_attention_bf16_kernel<VD><<<dim3((a.T + kTQ - 1) / kTQ, a.H, a.B), kTThreads, smem, st>>>(a, dk16, vec, qvec);
  return check_launch();
}

}  // namespace nb

using namespace nb;

extern "C" int nb_latent_prepare(const nb_latent_prepare_args* a, void* stream) {
  if (!a || !a->a || !a->cq || !a->q_norm || a->B < 1 || a->T < 1 || a->q_rank < 1 || a->q_off < 0 || a->ldcq < a->q_rank) return NB_ERR_ARG;
  if (a->dtype != NB_BF16 && a->dtype != NB_F32) return NB_ERR_ARG;
  if (a->q_off + a->q_rank > a->lda) return NB_ERR_SHAPE;
  if (a->kv_off >= 0) {
    if (!a->cache || !a->kv_norm || !a->cos2 || !a->sin2 || a->rank < 1 || a->rot < 0 || a->rot % 2 || a->ctx < 1 || a->pos0 < 0) return NB_ERR_ARG;
    if (a->kv_off + a->rank + a->rot > a->lda || a->ldc < a->rank + a->rot || a->pos0 + a->T > a->ctx) return NB_ERR_SHAPE;
  }
  if (int rc = check_device()) return rc;
  const dim3 grid((unsigned)a->B * a->T);
  const bool kv = a->kv_off >= 0;
  const bool vec = a->dtype == NB_BF16 && a->q_rank % 8 == 0 && a->q_off % 8 == 0 && a->lda % 8 == 0 && a->ldcq % 8 == 0 &&
                   a->q_rank <= 256 * kPvQ && (uintptr_t)a->a % 16 == 0 && (uintptr_t)a->cq % 16 == 0 && (uintptr_t)a->q_norm % 16 == 0 &&
                   (!kv || (a->kv_off % 8 == 0 && a->rank % 8 == 0 && a->rot % 8 == 0 && a->rank <= 256 * kPvQ && a->ldc % 8 == 0 &&
                            (uintptr_t)a->cache % 16 == 0 && (uintptr_t)a->kv_norm % 16 == 0 && (uintptr_t)a->cos2 % 16 == 0 &&
                            (uintptr_t)a->sin2 % 16 == 0));
  if (vec) {
    const int rows = a->B * a->T;
    return launch_pdl(latent_prepare_vec_kernel, dim3(((kv ? 2 : 1) * rows + 7) / 8), dim3(256), 0, (cudaStream_t)stream, *a, rows);
  }
  return a->dtype == NB_BF16 ? launch_pdl(latent_prepare_kernel<bf16>, grid, dim3(kPrepThreads), 0, (cudaStream_t)stream, *a)
                             : launch_pdl(latent_prepare_kernel<float>, grid, dim3(kPrepThreads), 0, (cudaStream_t)stream, *a);
}

extern "C" int nb_latent_attention(const nb_latent_attention_args* a, void* stream) {
  if (!a || !a->q || !a->kv || !a->cache || !a->out || !a->cos2 || !a->sin2 || a->B < 1 || a->T < 1 || a->H < 1 || a->dim < 1 || a->rot < 0 ||
      a->rot % 2 || a->vdim < 1 || a->pos0 < 0 || a->window < 0 || a->kv_pos0 < 0 || !(a->scale > 0.f))
    return NB_ERR_ARG;
  if (a->dtype != NB_BF16 && a->dtype != NB_F32) return NB_ERR_ARG;
  const int first = a->window > 0 ? std::max(0, a->pos0 - a->window + 1) : 0;
  if (a->pos0 + a->T > a->ctx || a->kv_pos0 > first || a->kv_pos0 + a->kv_rows < a->pos0 + a->T) return NB_ERR_SHAPE;
  if (a->ldq < a->H * (a->dim + a->rot) || a->ldo < a->H * a->vdim || a->ldc < a->rank + a->rot || a->v_off < a->H * a->dim ||
      a->ldkv < a->v_off + a->H * a->vdim || (a->gate && a->ldg < a->H))
    return NB_ERR_SHAPE;
  if (a->vdim > 256 || a->H > 65535 || a->B > 65535) return NB_ERR_SHAPE;
  if (int rc = check_device()) return rc;
  cudaStream_t st = (cudaStream_t)stream;
  if (a->dtype == NB_F32) return a->vdim <= 64 ? launch_latent_f32<8>(*a, st) : a->vdim <= 128 ? launch_latent_f32<16>(*a, st) : launch_latent_f32<32>(*a, st);
  return a->vdim <= 64    ? launch_latent_bf16<64>(*a, st)
         : a->vdim <= 128 ? launch_latent_bf16<128>(*a, st)
         : a->vdim <= 192 ? launch_latent_bf16<192>(*a, st)
                          : launch_latent_bf16<256>(*a, st);
}

extern "C" int nb_latent_decode(const nb_latent_decode_args* a, void* stream) {
  if (!a || !a->q || !a->a || !a->cache || !a->uk || !a->uv || !a->cos2 || !a->sin2 || !a->pos || !a->out || a->B < 1 || a->H < 1 || a->dim < 1 ||
      a->rot < 0 || a->rot % 2 || a->vdim < 1 || a->rank < 1 || a->ctx < 1 || a->window < 0 || (a->kv_off >= 0 && !a->kv_norm))
    return NB_ERR_ARG;
  if (a->cache_dtype != NB_BF16 && a->cache_dtype != NB_F32) return NB_ERR_ARG;
  if (a->ldq < a->H * (a->dim + a->rot) || a->ldo < a->H * a->vdim || a->ldc < a->rank + a->rot || a->ldu < a->rank || a->g_off < 0 ||
      a->g_off + a->H > a->lda || (a->kv_off >= 0 && a->kv_off + a->rank + a->rot > a->lda))
    return NB_ERR_SHAPE;
  if ((uintptr_t)a->cache % 16 || a->ldc % 8 || (uintptr_t)a->uk % 16 || (uintptr_t)a->uv % 16 || a->ldu % 8) return NB_ERR_ALIGN;
  if (a->H > 65535 || a->B > 65535) return NB_ERR_SHAPE;
  if (int rc = check_device()) return rc;
  if (a->rank > 4 * kLdThreads * kLdCols) return NB_ERR_SHAPE;
  const int want = 592 / std::max(1, a->B * a->H), S = want >= 8 ? 8 : want >= 4 ? 4 : want >= 2 ? 2 : 1;
  const int most = a->window > 0 ? std::min(a->window, a->ctx) : a->ctx;
  const int wide = a->cache_dtype == NB_F32;
  const int rdp = (a->rank + a->rot + 7) & ~7;
  const size_t row = (size_t)rdp * (wide ? 4 : 2);
  const int pper = ((a->rank + 1) / 2 + S - 1) / S, slot = (2 * pper + 2 + 3) & ~3;
  const size_t fixed = ((size_t)2 * rdp + ((a->dim + a->rot + 7) & ~7) + 2 * ((a->rot + 7) & ~7) + 4 * kLdThreads + S * slot + 4) * 4;
  if (fixed + 8 * (row + 4) > kLatentMaxSmem) return NB_ERR_SHAPE;
  // as many of a CTA's rows at a time as shared memory holds; two CTAs per SM when they do not all fit one each
  const size_t budget = (size_t)a->B * a->H * S > 112 && fixed + 8 * (row + 4) <= kLatentHalfSmem ? kLatentHalfSmem : kLatentMaxSmem;
  const int stage = (int)std::min<size_t>((most + S - 1) / S, (budget - fixed) / (row + 4));
  const size_t smem = fixed + (size_t)((stage + 3) & ~3) * 4 + stage * row;
  static bool done[2][64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  auto kernel = wide ? latent_decode_kernel<float> : latent_decode_kernel<bf16>;
  if (!done[wide][dev & 63]) {
    if (cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLatentMaxSmem + 64)) return record_cuda_error(e);
    done[wide][dev & 63] = true;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(a->H, a->B, S);
  cfg.blockDim = dim3(kLdThreads);
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
  return record_cuda_error(cudaLaunchKernelEx(&cfg, kernel, *a, stage));
}
