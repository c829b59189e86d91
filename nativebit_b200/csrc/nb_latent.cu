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

__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)) : "memory");
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)) : "memory");
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&h);
}

template <int VD>
__global__ void __launch_bounds__(kTThreads) latent_attention_bf16_kernel(const nb_latent_attention_args p, int dk16, int vec) {
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
      const int nd = p.dim >> 3, nr = p.rot >> 3, nk = nd + nr, nv = p.vdim >> 3;
      for (int i = tid; i < kTK * (nk + nv); i += kTThreads) {
        const int j = i / (nk + nv), c = i - j * (nk + nv), pos = k0 + j;
        bf16* dst = c < nk ? kd + j * dkp + c * 8 : vd + j * vp + (c - nk) * 8;
        if (pos <= last) {
          const bf16* row = kv + (size_t)(pos - p.kv_pos0) * p.ldkv;
          const bf16* src = c < nd ? row + h * p.dim + c * 8
                            : c < nk ? cache + (size_t)pos * p.ldc + p.rank + (c - nd) * 8
                                     : row + p.v_off + h * p.vdim + (c - nk) * 8;
          cp16(dst, src);
        } else {
          *reinterpret_cast<uint4*>(dst) = make_uint4(0u, 0u, 0u, 0u);
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
  copy_tile(0, 0);
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

  // this lane's two rows of the warp's 16 queries: lane / 4 and lane / 4 + 8
  const int rowa = warp * 16 + (lane >> 2);
  const int pos_a = p.pos0 + min(q0 + rowa, p.T - 1), pos_b = p.pos0 + min(q0 + rowa + 8, p.T - 1);
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
    float na = ma, nb_ = mb;
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int pos = k0 + n * 8 + (lane & 3) * 2 + (j & 1), me = j < 2 ? pos_a : pos_b;
        const bool seen = pos <= me && (p.window <= 0 || me - pos < p.window);
        s[n][j] = seen ? s[n][j] * sl2 : -INFINITY;
        if (j < 2) na = fmaxf(na, s[n][j]);
        else nb_ = fmaxf(nb_, s[n][j]);
      }
#pragma unroll
    for (int x = 1; x < 4; x <<= 1) {
      na = fmaxf(na, __shfl_xor_sync(0xffffffffu, na, x));
      nb_ = fmaxf(nb_, __shfl_xor_sync(0xffffffffu, nb_, x));
    }
    const float ba = na == -INFINITY ? 0.f : na, bb_ = nb_ == -INFINITY ? 0.f : nb_;   // nothing seen yet: all weights are 0
    const float ca = exp2f(ma - ba), cb = exp2f(mb - bb_);
    ma = na; mb = nb_;
    la *= ca; lb *= cb;
#pragma unroll
    for (int i = 0; i < VD / 8; ++i) { o[i][0] *= ca; o[i][1] *= ca; o[i][2] *= cb; o[i][3] *= cb; }
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      s[n][0] = exp2f(s[n][0] - ba); s[n][1] = exp2f(s[n][1] - ba);
      s[n][2] = exp2f(s[n][2] - bb_); s[n][3] = exp2f(s[n][3] - bb_);
      la += s[n][0] + s[n][1];
      lb += s[n][2] + s[n][3];
    }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {                   // 16 keys per step
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {                    // registers of the A fragment: (row a, keys 0-7), (row b, ..), (row a, keys 8-15), (row b, ..)
        const float x = s[2 * kk + (j >> 1)][(j & 1) * 2], y = s[2 * kk + (j >> 1)][(j & 1) * 2 + 1];
        hi[j] = pack_bf16(x, y);
        lo[j] = pack_bf16(x - bf_lo(hi[j]), y - bf_hi(hi[j]));
      }
#pragma unroll
      for (int n = 0; n < VD / 16; ++n) {
        uint32_t bb[4];
        ldsm_x4_t(bb, vt + (kk * 16 + (lane & 15)) * vp + n * 16 + (lane >> 4) * 8);
        mma_bf16(o[2 * n], hi, bb[0], bb[1]);
        mma_bf16(o[2 * n + 1], hi, bb[2], bb[3]);
        mma_bf16(o[2 * n], lo, bb[0], bb[1]);
        mma_bf16(o[2 * n + 1], lo, bb[2], bb[3]);
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
// weighted latent, slices of the values for W_uv; the slices travel through distributed shared memory.
constexpr int kLdThreads = 256, kLdWarps = kLdThreads / 32;

template <typename T>
__global__ void __launch_bounds__(kLdThreads) latent_decode_kernel(const nb_latent_decode_args p) {
  extern __shared__ __align__(16) float dsm[];
  __shared__ float red[2 * kLdWarps], red2[kLdWarps], red3[kLdWarps];
  cg::cluster_group cluster = cg::this_cluster();
  const int S = (int)cluster.num_blocks(), rank_id = (int)cluster.block_rank();
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int rd = p.rank + p.rot, dk = p.dim + p.rot, rdp = (rd + 7) & ~7;
  float* qa = dsm;                     // [rdp] q' and the rotated query part: what the cached rows are multiplied with
  float* row = qa + rdp;               // [rdp] this position's row of the cache
  float* ol = row + rdp;               // [rdp] weighted latent of this CTA's keys, then of all
  float* xch = ol + rdp;               // [rdp + 8] what the other CTAs read: weighted latent, maximum, sum
  float* qn = xch + rdp + 8;           // [dk] this head's query
  float* part = qn + ((dk + 7) & ~7);  // [kLdThreads * 2] partial sums
  float* sc = part + 2 * kLdThreads;   // scores of this CTA's keys
  pdl_enter();
  const long long pos = *p.pos;
  if (pos < 0 || pos >= p.ctx) return; // the same for every CTA
  const int n = p.window > 0 ? min((int)pos + 1, p.window) : (int)pos + 1, first = (int)pos + 1 - n;
  const int per = (n + S - 1) / S, k0 = first + rank_id * per, cnt = max(0, min(first + n, k0 + per) - k0);
  T* cache = reinterpret_cast<T*>(p.cache) + (size_t)b * p.ctx * p.ldc;
  const float *cs = p.cos2 + (size_t)pos * p.rot, *sn = p.sin2 + (size_t)pos * p.rot;

  for (int i = tid; i < dk; i += kLdThreads) qn[i] = p.q[(size_t)b * p.ldq + h * dk + i];
  for (int i = rd + tid; i < rdp; i += kLdThreads) { qa[i] = 0.f; row[i] = 0.f; }
  if (p.kv_off >= 0) {
    const float* kv = p.a + (size_t)b * p.lda + p.kv_off;
    float mean, inv;
    norm_stats<kLdWarps>(NB_NORM_RMS, p.rank, p.eps, red,
                         [&](auto f) { for (int i = tid; i < p.rank; i += kLdThreads) f(kv[i]); }, mean, inv);
    T* crow = cache + (size_t)pos * p.ldc;
    for (int i = tid; i < rd; i += kLdThreads) {
      const T v = from_f<T>(i < p.rank ? kv[i] * inv * p.kv_norm[i] : rotated([&](int j) { return kv[p.rank + j]; }, cs, sn, i - p.rank));
      row[i] = to_f(v);
      if (h == 0 && rank_id == 0) crow[i] = v;
    }
  } else {
    for (int i = tid; i < rd; i += kLdThreads) row[i] = to_f(cache[(size_t)pos * p.ldc + i]);
  }
  cluster.sync();                      // every CTA of the cluster runs: its shared memory may be written from here on
  for (int d = tid; d < p.rot; d += kLdThreads) qa[p.rank + d] = rotated([&](int j) { return qn[p.dim + j]; }, cs, sn, d);

  // q'[j] = sum_d W_uk[h][d][j] q[d] for this CTA's slice of j (pairs), the d range split over groups of threads
  const int pairs = (p.rank + 1) / 2, pper = (pairs + S - 1) / S, p0 = rank_id * pper, pn = max(0, min(pairs, p0 + pper) - p0);
  {
    const bf16* uk = reinterpret_cast<const bf16*>(p.uk) + (size_t)h * p.dim * p.ldu;
    for (int base = 0; base < pn; base += kLdThreads) {
      const int cols = min(pn - base, kLdThreads), groups = kLdThreads / cols, gi = tid / cols, c = tid - gi * cols;
      float x = 0.f, y = 0.f;
      if (gi < groups) {
        const int j = 2 * (p0 + base + c);
#pragma unroll 8
        for (int d = gi; d < p.dim; d += groups) {
          const uint32_t w = *reinterpret_cast<const uint32_t*>(uk + (size_t)d * p.ldu + j);
          x = fmaf(bf_lo(w), qn[d], x);
          y = fmaf(bf_hi(w), qn[d], y);
        }
      }
      part[2 * tid] = x; part[2 * tid + 1] = y;
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
  }
  cluster.sync();

  // scores: a warp takes a key at a time, eight columns per lane and step
  float mx = -FLT_MAX;
  for (int j = warp; j < cnt; j += kLdWarps) {
    float s = 0.f;
    if (k0 + j == (int)pos) {
      for (int i = lane; i < rd; i += 32) s = fmaf(row[i], qa[i], s);
    } else {
      const T* cr = cache + (size_t)(k0 + j) * p.ldc;
      if (sizeof(T) == 2) {
        for (int i = lane * 8; i < rd; i += 256) {
          const uint4 t = *reinterpret_cast<const uint4*>(cr + i);   // ldc is a multiple of 8; past rd qa is zero
          const float4 a = *reinterpret_cast<const float4*>(qa + i), c = *reinterpret_cast<const float4*>(qa + i + 4);
          const uint32_t u[4] = {t.x, t.y, t.z, t.w};
          const float q8[8] = {a.x, a.y, a.z, a.w, c.x, c.y, c.z, c.w};
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            if (i + 2 * e < rd) s = fmaf(bf_lo(u[e]), q8[2 * e], s);
            if (i + 2 * e + 1 < rd) s = fmaf(bf_hi(u[e]), q8[2 * e + 1], s);
          }
        }
      } else {
        for (int i = lane; i < rd; i += 32) s = fmaf(to_f(cr[i]), qa[i], s);
      }
    }
    s = warp_sum(s) * p.scale;
    if (lane == 0) sc[j] = s;
    mx = fmaxf(mx, s);
  }
  if (lane == 0) red2[warp] = mx;
  __syncthreads();
  mx = red2[0];
#pragma unroll
  for (int i = 1; i < kLdWarps; ++i) mx = fmaxf(mx, red2[i]);
  float sum = 0.f;
  for (int j = tid; j < cnt; j += kLdThreads) {
    const float e = expf(sc[j] - mx);
    sc[j] = e;
    sum += e;
  }
  const float tot = block_sum<kLdWarps>(sum, red3);    // its barrier also publishes sc

  // weighted latent of this CTA's keys: pairs of columns per thread, the keys split over groups of threads
  for (int base = 0; base < pairs; base += kLdThreads) {
    const int cols = min(pairs - base, kLdThreads), groups = kLdThreads / cols, gi = tid / cols, c = tid - gi * cols;
    float x = 0.f, y = 0.f;
    if (gi < groups) {
      const int i = 2 * (base + c);
#pragma unroll 4
      for (int j = gi; j < cnt; j += groups) {
        const float w = sc[j];
        if (k0 + j == (int)pos) {
          x = fmaf(w, row[i], x);
          y = fmaf(w, row[i + 1], y);
        } else if (sizeof(T) == 2) {
          const uint32_t t = *reinterpret_cast<const uint32_t*>(cache + (size_t)(k0 + j) * p.ldc + i);
          x = fmaf(w, bf_lo(t), x);
          y = fmaf(w, bf_hi(t), y);
        } else {
          const float2 t = *reinterpret_cast<const float2*>(cache + (size_t)(k0 + j) * p.ldc + i);
          x = fmaf(w, t.x, x);
          y = fmaf(w, t.y, y);
        }
      }
    }
    part[2 * tid] = x; part[2 * tid + 1] = y;
    __syncthreads();
    for (int i = tid; i < 2 * cols; i += kLdThreads) {
      float v = 0.f;
      for (int g = 0; g < groups; ++g) v += part[2 * g * cols + i];
      xch[2 * base + i] = v;
    }
    __syncthreads();
  }
  if (tid == 0) { xch[rdp] = mx; xch[rdp + 1] = tot; }
  cluster.sync();
  // this CTA's slice of the merged latent, to everyone
  {
    float m_all = -FLT_MAX, den = 0.f;
    for (int r = 0; r < S; ++r) m_all = fmaxf(m_all, cluster.map_shared_rank(xch, r)[rdp]);
    for (int r = 0; r < S; ++r) {      // a CTA without keys has maximum -FLT_MAX and sum 0
      const float* rx = cluster.map_shared_rank(xch, r);
      den += expf(rx[rdp] - m_all) * rx[rdp + 1];
    }
    for (int i = 2 * p0 + tid; i < min(p.rank, 2 * (p0 + pn)); i += kLdThreads) {
      float num = 0.f;
      for (int r = 0; r < S; ++r) {
        const float* rx = cluster.map_shared_rank(xch, r);
        num += expf(rx[rdp] - m_all) * rx[i];
      }
      const float v = num / den;
      for (int r = 0; r < S; ++r) cluster.map_shared_rank(ol, r)[i] = v;
    }
  }
  cluster.sync();                      // also: nobody reads another CTA's shared memory after this
  const int vper = (p.vdim + S - 1) / S, v0 = rank_id * vper, v1 = min(p.vdim, v0 + vper);
  const float g = sigmoid_f(p.a[(size_t)b * p.lda + p.g_off + h]);
  for (int v = v0 + warp; v < v1; v += kLdWarps) {
    const bf16* uv = reinterpret_cast<const bf16*>(p.uv) + (size_t)(h * p.vdim + v) * p.ldu;
    float s = 0.f;
    for (int i = lane * 2; i < p.rank; i += 64) {
      const uint32_t w = *reinterpret_cast<const uint32_t*>(uv + i);
      s = fmaf(bf_lo(w), ol[i], s);
      if (i + 1 < p.rank) s = fmaf(bf_hi(w), ol[i + 1], s);
    }
    s = warp_sum(s);
    if (lane == 0) p.out[(size_t)b * p.ldo + h * p.vdim + v] = s * g;
  }
}

constexpr size_t kLatentMaxSmem = 200 * 1024;

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
  latent_attention_bf16_kernel<VD><<<dim3((a.T + kTQ - 1) / kTQ, a.H, a.B), kTThreads, smem, st>>>(a, dk16, vec);
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
  return a->dtype == NB_BF16 ? launch_pdl(latent_prepare_kernel<bf16>, grid, dim3(kPrepThreads), 0, (cudaStream_t)stream, *a)
                             : launch_pdl(latent_prepare_kernel<float>, grid, dim3(kPrepThreads), 0, (cudaStream_t)stream, *a);
}

extern "C" int nb_latent_attention(const nb_latent_attention_args* a, void* stream) {
  if (!a || !a->q || !a->kv || !a->cache || !a->out || !a->cos2 || !a->sin2 || a->B < 1 || a->T < 1 || a->H < 1 || a->dim < 1 || a->rot < 0 ||
      a->rot % 2 || a->vdim < 1 || a->pos0 < 0 || a->window < 0 || a->kv_pos0 < 0)
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
  const int want = 592 / std::max(1, a->B * a->H), S = want >= 8 ? 8 : want >= 4 ? 4 : want >= 2 ? 2 : 1;
  const int most = a->window > 0 ? std::min(a->window, a->ctx) : a->ctx;
  const int rdp = (a->rank + a->rot + 7) & ~7;
  const size_t smem = ((size_t)4 * rdp + 8 + ((a->dim + a->rot + 7) & ~7) + 2 * kLdThreads + (most + S - 1) / S + 8) * 4;
  if (smem > kLatentMaxSmem) return NB_ERR_SHAPE;
  static bool done[2][64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  const int wide = a->cache_dtype == NB_F32;
  auto kernel = wide ? latent_decode_kernel<float> : latent_decode_kernel<bf16>;
  if (!done[wide][dev & 63]) {
    if (cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLatentMaxSmem)) return record_cuda_error(e);
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
  return record_cuda_error(cudaLaunchKernelEx(&cfg, kernel, *a));
}
