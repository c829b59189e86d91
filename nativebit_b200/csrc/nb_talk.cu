// Grouped attention over a sliding window whose scores pass through a soft cap, a penalty that grows with the distance and
// a mixing of the heads (s'_h = sum_g talk[h][g] s_g) before the softmax, with an output gate per element.
//
//   nb_cache_append     keys and values of a portion into the cache
//   nb_talk_attention   a portion of a prompt, in two kernels per block of queries: the mixed scores of all heads (a head's
//                       softmax needs every head's scores of a pair), then softmax and values per head
//   nb_talk_decode      one position per sequence: a cluster of CTAs shares the keys, every CTA takes all heads of its keys
#include <cuda_runtime.h>
#include <cuda_bf16.h>
#include <cooperative_groups.h>

#include <algorithm>
#include <cfloat>

#include "nb_layered.cuh"
#include "nb_mma.cuh"

namespace nb {

namespace cg = cooperative_groups;

__global__ void __launch_bounds__(256) cache_append_kernel(const uint4* __restrict__ src, int ld16, int off16, int n16, uint4* __restrict__ cache,
                                                           int ldc16, int T, int ctx, int pos0, long long total) {
  pdl_enter();
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= total) return;
  const int row = (int)(i / n16), c = (int)(i - (long long)row * n16), b = row / T, t = row - b * T;
  cache[((size_t)b * ctx + pos0 + t) * ldc16 + c] = src[(size_t)row * ld16 + off16 + c];
}

// ---- mixed scores.  Queries come in tiles of 64; a tile's keys are the `span` positions from first_key() on, and the
// workspace holds [sequence][tile of the block][head][64][span rounded up to 64], unseen pairs as -infinity.
constexpr int kQT = 64, kKT = 64;

struct TalkBlock {
  float* ws;
  int tile0, tiles, ld;                  // first query tile of the block, tiles in it, row length
};

__host__ __device__ inline int talk_first_key(int pos0, int q0, int window) {
  const int f = pos0 + q0 - window + 1;
  return window > 0 && f > 0 ? f : 0;
}

__device__ __forceinline__ float soft_cap_fast(float x, float cap2, float cap) {    // cap * tanh(x), cap2 = 2 log2(e) folded into x's factor
  return cap - __fdividef(2.f * cap, 1.f + ex2(x * cap2));
}

// bf16.  A CTA of eight warps owns 16 queries, whose rows of all heads stay in shared memory, and walks `chunk` steps of
// 64 NB keys; a step's keys arrive one key/value head at a time through a ring of `stages`.  A warp takes 8 NB of the keys:
// the raw scores of every head of a pair stay in the registers of one thread, where the heads are mixed.  HM >= H;
// kTwo: two heads of a group at a time share the key fragments (an even number of heads per group).
constexpr int kScThreads = 256, kSq = 16;

template <int HM, int NB, bool kTwo>
__global__ void __launch_bounds__(kScThreads, 1) talk_scores_bf16_kernel(const nb_talk_attention_args p, TalkBlock blk, int dk16, int chunk, int stages,
                                                                         int vec) {
  extern __shared__ __align__(16) bf16 tsm[];
  constexpr int KW = 64 * NB, kPen = kSq + KW, R = kTwo ? 2 : 1;
  const int dkp = dk16 + 8, H = p.H, D = p.dim, rep = H / p.G;
  bf16* q_s = tsm;                       // [H][16][dkp]
  bf16* k_s = q_s + H * kSq * dkp;       // [stages][KW][dkp]
  float* talk_s = reinterpret_cast<float*>(k_s + stages * KW * dkp);   // [H][HM]
  float* pen_s = talk_s + H * HM;        // [H][kPen]: of a step, by distance from its smallest
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int sub = gridDim.y - 1 - blockIdx.y, local = sub / (kQT / kSq), r0 = (sub & (kQT / kSq - 1)) * kSq, b = blockIdx.z;   // longest first
  const int q0 = (blk.tile0 + local) * kQT;
  const int first = talk_first_key(p.pos0, q0, p.window), last = p.pos0 + min(q0 + kQT - 1, p.T - 1);
  const int span = ((last - first) / kKT + 1) * kKT;               // what the tile's readers take
  const int c0 = blockIdx.x * chunk * KW, steps = min(chunk, (span - c0 + KW - 1) / KW);
  if (steps <= 0 || q0 + r0 >= p.T) return;
  const bf16* q = reinterpret_cast<const bf16*>(p.q);
  const bf16* cache = reinterpret_cast<const bf16*>(p.cache) + (size_t)b * p.ctx * p.ldc;
  for (int i = tid; i < (H * kSq + stages * KW) * (dkp - D); i += kScThreads) {      // columns past dim stay zero
    const int r = i / (dkp - D);
    q_s[r * dkp + D + i - r * (dkp - D)] = from_f<bf16>(0.f);
  }
  for (int i = tid; i < H * HM; i += kScThreads) {
    const int h = i / HM, g = i - h * HM;
    talk_s[i] = g < H ? p.talk[h * H + g] : 0.f;
  }
  auto copy = [&](bf16* dst, int rows, auto row_of) {
    if (vec) {
      const int c8 = (tid & 7) * 8;
      for (int r = tid >> 3; r < rows; r += kScThreads / 8) {
        const bf16* src = row_of(r);
        for (int c = c8; c < D; c += 64) {
          if (src) cp16(dst + r * dkp + c, src + c);
          else *reinterpret_cast<uint4*>(dst + r * dkp + c) = make_uint4(0u, 0u, 0u, 0u);
        }
      }
    } else {
      for (int i = tid; i < rows * D; i += kScThreads) {
        const int r = i / D, c = i - r * D;
        const bf16* src = row_of(r);
        dst[r * dkp + c] = src ? src[c] : from_f<bf16>(0.f);
      }
    }
  };
  const int items = steps * p.G;         // (step, key/value head) in order; item i uses stage i % stages
  int ni = 0, ng = 0, ns = 0, nk = first + c0;                     // next item to request: its number, head, stage, first key
  auto fetch = [&]() {
    if (ni < items) {
      const int g = ng, k0 = nk;
      copy(k_s + ns * KW * dkp, KW, [&](int r) { return k0 + r <= last ? cache + (size_t)(k0 + r) * p.ldc + g * D : nullptr; });
      ++ni;
      if (++ng == p.G) { ng = 0; nk += KW; }
      if (++ns == stages) ns = 0;
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto penalties = [&](int k0) {
    const int dmin = p.pos0 + q0 + r0 - (k0 + KW - 1);
    for (int i = tid; i < H * kPen; i += kScThreads) {
      const int h = i / kPen, d = dmin + i - h * kPen;
      pen_s[i] = p.penalty && d >= 0 && d < p.n_pen ? p.penalty[(size_t)h * p.n_pen + d] : 0.f;
    }
  };
  copy(q_s, H * kSq, [&](int r) { return q + (size_t)(b * p.T + min(q0 + r0 + (r & (kSq - 1)), p.T - 1)) * p.ldq + (r / kSq) * D; });
  for (int i = 0; i + 1 < stages; ++i) fetch();                    // the queries travel with the first
  penalties(first + c0);
  const int rowa = lane >> 2, kc = warp * 8 * NB + (lane & 3) * 2; // this lane's first query row and key column
  const float sx = p.softcap > 0.f ? p.scale / p.softcap : p.scale, cap2 = 2.f * 1.4426950408889634f;
  const int pa = p.pos0 + q0 + r0 + rowa, plast = p.pos0 + p.T - 1;
  float* ws = blk.ws + ((size_t)(b * blk.tiles + local) * H * kQT + r0 + rowa) * blk.ld + kc;
  int st = 0, left = 0;                  // stage of the current key/value head, heads of its group still to come
  for (int step = 0; step < steps; ++step) {
    const int k0 = first + c0 + step * KW;
    float s[HM][NB][4];
#pragma unroll
    for (int h = 0; h < HM; h += R) {
#pragma unroll
      for (int r = 0; r < R; ++r)
#pragma unroll
        for (int n = 0; n < NB; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[h + r][n][e] = 0.f;
      if (h < H) {                       // block-uniform
        if (left == 0) {                 // a group begins: its keys are there, and the stage before may be filled again
          if (stages == 3) asm volatile("cp.async.wait_group 1;" ::: "memory");
          else asm volatile("cp.async.wait_group 0;" ::: "memory");
          __syncthreads();
          fetch();
          left = rep;
        }
        left -= R;
        const bf16* qt = q_s + h * kSq * dkp + (lane & 15) * dkp + (lane >> 4) * 8;
        const bf16* kt = k_s + (st * KW + warp * 8 * NB) * dkp;
#pragma unroll 4
        for (int kk = 0; kk < dk16; kk += 16) {
          uint32_t a[R][4], bb[(NB + 1) / 2][4];
#pragma unroll
          for (int r = 0; r < R; ++r) ldsm_x4(a[r], qt + r * kSq * dkp + kk);
#pragma unroll
          for (int n = 0; n < NB; n += 2)          // with eight keys per warp the other half of the load is not used
            ldsm_x4(bb[n / 2], kt + (n * 8 + (lane & 7) + (NB > 1 ? (lane >> 4) << 3 : 0)) * dkp + kk + ((lane >> 3) & 1) * 8);
#pragma unroll
          for (int n = 0; n < NB; ++n)
#pragma unroll
            for (int r = 0; r < R; ++r) mma_bf16(s[h + r][n], a[r], bb[n / 2][(n & 1) * 2], bb[n / 2][(n & 1) * 2 + 1]);
        }
        if (left == 0 && ++st == stages) st = 0;
#pragma unroll
        for (int r = 0; r < R; ++r) {
          // the distance is (r0 + row) - (k0 + key), from the step's smallest on
          const float* pen = pen_s + (h + r) * kPen + rowa + KW - 1 - kc;
#pragma unroll
          for (int n = 0; n < NB; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float x = s[h + r][n][e] * sx;
              s[h + r][n][e] = (p.softcap > 0.f ? soft_cap_fast(x, cap2, p.softcap) : x) - pen[(e >> 1) * 8 - n * 8 - (e & 1)];
            }
        }
      }
    }
    if (step + 1 < steps) {
      __syncthreads();                   // nobody reads this step's penalties any more; the next group's barrier publishes the new ones
      penalties(k0 + KW);
    }
    if (k0 - first + warp * 8 * NB < span) {       // mix and store; a tile's rows end with its span
      bool seen[NB][4];
#pragma unroll
      for (int n = 0; n < NB; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int pos = k0 + kc + n * 8 + (e & 1), me = min(pa + (e >> 1) * 8, plast);
          seen[n][e] = pos <= me && (p.window <= 0 || me - pos < p.window);
        }
      float* dst = ws + (k0 - first);
      for (int h = 0; h < H; ++h) {
        float m[NB][4];
#pragma unroll
        for (int n = 0; n < NB; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) m[n][e] = 0.f;
#pragma unroll
        for (int g = 0; g < HM; g += 2) {
          const float2 t = *reinterpret_cast<const float2*>(talk_s + h * HM + g);
#pragma unroll
          for (int n = 0; n < NB; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) m[n][e] = fmaf(t.x, s[g][n][e], fmaf(t.y, s[g + 1][n][e], m[n][e]));
        }
#pragma unroll
        for (int n = 0; n < NB; ++n) {
          *reinterpret_cast<float2*>(dst + n * 8) = make_float2(seen[n][0] ? m[n][0] : -INFINITY, seen[n][1] ? m[n][1] : -INFINITY);
          *reinterpret_cast<float2*>(dst + (size_t)8 * blk.ld + n * 8) = make_float2(seen[n][2] ? m[n][2] : -INFINITY, seen[n][3] ? m[n][3] : -INFINITY);
        }
        dst += (size_t)kQT * blk.ld;
      }
    }
  }
}

// Any dtype, fp32 multiply-adds: 16 queries x 16 keys of all heads per CTA, one pair per thread; the raw scores of a pair wait
// in a shared-memory column of its own.
constexpr int kSt = 16, kSd = 64;

template <typename T> __global__ void __launch_bounds__(256) talk_scores_kernel(const nb_talk_attention_args p, TalkBlock blk) {
  extern __shared__ __align__(16) float ssm[];
  __shared__ float qs[kSt][kSd + 1], ks[kSt][kSd + 1];
  float* raw = ssm;                      // [H][256]
  float* talk_s = raw + p.H * 256;       // [H][H]
  const int tid = threadIdx.x, ty = tid >> 4, tx = tid & 15;
  const int local = blockIdx.y >> 2, tile = blk.tile0 + local, q0 = tile * kQT, r0 = (blockIdx.y & 3) * kSt, b = blockIdx.z;
  const int first = talk_first_key(p.pos0, q0, p.window), last = p.pos0 + min(q0 + kQT - 1, p.T - 1);
  const int k0 = first + blockIdx.x * kSt;
  if (k0 >= first + ((last - first) / kKT + 1) * kKT) return;
  const int rep = p.H / p.G, D = p.dim;
  const T* q = reinterpret_cast<const T*>(p.q);
  const T* cache = reinterpret_cast<const T*>(p.cache) + (size_t)b * p.ctx * p.ldc;
  for (int i = tid; i < p.H * p.H; i += 256) talk_s[i] = p.talk[i];
  const int me = p.pos0 + min(q0 + r0 + ty, p.T - 1), pos = k0 + tx;
  const bool seen = pos <= me && (p.window <= 0 || me - pos < p.window);
  for (int h = 0; h < p.H; ++h) {
    float x = 0.f;
    for (int d0 = 0; d0 < D; d0 += kSd) {
      __syncthreads();                   // the piece before is no longer read
      for (int i = tid; i < kSt * kSd; i += 256) {
        const int r = i / kSd, d = d0 + (i & (kSd - 1));
        qs[r][i & (kSd - 1)] = d < D ? to_f(q[(size_t)(b * p.T + min(q0 + r0 + r, p.T - 1)) * p.ldq + h * D + d]) : 0.f;
        ks[r][i & (kSd - 1)] = d < D && k0 + r <= last ? to_f(cache[(size_t)(k0 + r) * p.ldc + (h / rep) * D + d]) : 0.f;
      }
      __syncthreads();
      const int dn = min(kSd, D - d0);
      for (int d = 0; d < dn; ++d) x = fmaf(qs[ty][d], ks[tx][d], x);
    }
    x *= p.scale;
    if (p.softcap > 0.f) x = p.softcap * tanhf(x / p.softcap);
    if (p.penalty && seen) x -= p.penalty[(size_t)h * p.n_pen + me - pos];
    raw[h * 256 + tid] = x;
  }
  __syncthreads();
  float* ws = blk.ws + ((size_t)(b * blk.tiles + local) * p.H * kQT + r0 + ty) * blk.ld + blockIdx.x * kSt + tx;
  for (int h = 0; h < p.H; ++h) {
    float m = 0.f;
    for (int g = 0; g < p.H; ++g) m = fmaf(talk_s[h * p.H + g], raw[g * 256 + tid], m);
    ws[(size_t)h * kQT * blk.ld] = seen ? m : -INFINITY;
  }
}

// ---- softmax over the mixed scores and the weighted values, bf16: 64 queries x at most VD value columns of a head per CTA,
// four warps, values in tiles of 64 keys through two stages; a lane reads the scores it multiplies straight from the
// workspace, one tile ahead.
constexpr int kPvThreads = 128;

template <int VD>
__global__ void __launch_bounds__(kPvThreads, VD <= 128 ? 3 : 1) talk_values_bf16_kernel(const nb_talk_attention_args p, TalkBlock blk, int vtiles, int vec) {
  extern __shared__ __align__(16) bf16 v_s[];   // [2][64][VD + 8]
  constexpr int vp = VD + 8;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.x / vtiles, v0 = (blockIdx.x - h * vtiles) * VD, vn = min(VD, p.vdim - v0), b = blockIdx.z;
  const int local = gridDim.y - 1 - blockIdx.y, q0 = (blk.tile0 + local) * kQT;    // longest first
  const int first = talk_first_key(p.pos0, q0, p.window), last = p.pos0 + min(q0 + kQT - 1, p.T - 1), tiles = (last - first) / kKT + 1;
  const bf16* vals = reinterpret_cast<const bf16*>(p.cache) + (size_t)b * p.ctx * p.ldc + p.v_off + (h / (p.H / p.G)) * p.vdim + v0;
  for (int i = tid; i < 2 * kKT * (vp - vn); i += kPvThreads) {    // columns past the values stay zero
    const int r = i / (vp - vn);
    v_s[r * vp + vn + i - r * (vp - vn)] = from_f<bf16>(0.f);
  }
  auto copy_tile = [&](int t, int st) {
    const int k0 = first + t * kKT;
    bf16* vd = v_s + st * kKT * vp;
    if (vec) {
      const int c8 = (tid & 7) * 8;
#pragma unroll
      for (int jr = 0; jr < kKT; jr += kPvThreads / 8) {
        const int j = jr + (tid >> 3), pos = k0 + j;
        bf16* vr = vd + j * vp;
        for (int c = c8; c < vn; c += 64) {
          if (pos <= last) cp16(vr + c, vals + (size_t)pos * p.ldc + c);
          else *reinterpret_cast<uint4*>(vr + c) = make_uint4(0u, 0u, 0u, 0u);
        }
      }
    } else {
      for (int i = tid; i < kKT * vn; i += kPvThreads) {
        const int j = i / vn, c = i - j * vn, pos = k0 + j;
        vd[j * vp + c] = pos <= last ? vals[(size_t)pos * p.ldc + c] : from_f<bf16>(0.f);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  copy_tile(0, 0);
  const int rowa = warp * 16 + (lane >> 2), c2 = (lane & 3) * 2;
  const float* ws = blk.ws + (((size_t)(b * blk.tiles + local) * p.H + h) * kQT + rowa) * blk.ld + c2;
  const size_t row8 = (size_t)8 * blk.ld;
  float2 nx[8][2];                       // the next tile's scores: rows a and b, eight pairs of keys
  auto load_scores = [&](int t) {
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      nx[n][0] = __ldcs(reinterpret_cast<const float2*>(ws + t * kKT + n * 8));
      nx[n][1] = __ldcs(reinterpret_cast<const float2*>(ws + row8 + t * kKT + n * 8));
    }
  };
  load_scores(0);
  constexpr float kLog2e = 1.4426950408889634f;
  float o[VD / 8][4];
#pragma unroll
  for (int i = 0; i < VD / 8; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) o[i][j] = 0.f;
  float ma = -INFINITY, mb = -INFINITY, la = 0.f, lb = 0.f;
  for (int t = 0; t < tiles; ++t) {
    const int st = t & 1;
    float s[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n) { s[n][0] = nx[n][0].x; s[n][1] = nx[n][0].y; s[n][2] = nx[n][1].x; s[n][3] = nx[n][1].y; }
    if (t + 1 < tiles) {
      load_scores(t + 1);
      copy_tile(t + 1, st ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
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
    const float ba = na == -INFINITY ? 0.f : na, bb_ = nb_ == -INFINITY ? 0.f : nb_;   // nothing seen yet: all weights are 0
    const float ca = ex2((ma - ba) * kLog2e), cb = ex2((mb - bb_) * kLog2e);
    ma = na; mb = nb_;
    la *= ca; lb *= cb;
#pragma unroll
    for (int i = 0; i < VD / 8; ++i) { o[i][0] *= ca; o[i][1] *= ca; o[i][2] *= cb; o[i][3] *= cb; }
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      s[n][0] = ex2((s[n][0] - ba) * kLog2e); s[n][1] = ex2((s[n][1] - ba) * kLog2e);
      s[n][2] = ex2((s[n][2] - bb_) * kLog2e); s[n][3] = ex2((s[n][3] - bb_) * kLog2e);
      la += s[n][0] + s[n][1];
      lb += s[n][2] + s[n][3];
    }
    __syncthreads();                     // the tile's values
    const bf16* vt = v_s + st * kKT * vp;
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {     // 16 keys per step
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) split_bf16(s[2 * kk + (j >> 1)][(j & 1) * 2], s[2 * kk + (j >> 1)][(j & 1) * 2 + 1], hi[j], lo[j]);
#pragma unroll
      for (int n = 0; n < VD / 16; n += 2) {     // four independent products before an accumulator comes again
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
    __syncthreads();                     // before the stage is filled again
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
    const float f = 1.f / (half ? lb : la);
    const bf16* gate = p.gate ? reinterpret_cast<const bf16*>(p.gate) + row * p.ldg + h * p.vdim + v0 : nullptr;
    bf16* out = reinterpret_cast<bf16*>(p.out) + row * p.ldo + h * p.vdim + v0;
#pragma unroll
    for (int i = 0; i < VD / 8; ++i) {
      const int d = i * 8 + c2;
      float x = o[i][2 * half] * f, y = o[i][2 * half + 1] * f;
      if (vec) {
        if (d < vn) {
          if (gate) {
            const uint32_t g = *reinterpret_cast<const uint32_t*>(gate + d);
            x *= __fdividef(1.f, 1.f + __expf(-bf_lo(g)));
            y *= __fdividef(1.f, 1.f + __expf(-bf_hi(g)));
          }
          *reinterpret_cast<uint32_t*>(out + d) = pack_bf16(x, y);
        }
      } else {
        if (d < vn) out[d] = from_f<bf16>(gate ? x * sigmoid_f(to_f(gate[d])) : x);
        if (d + 1 < vn) out[d + 1] = from_f<bf16>(gate ? y * sigmoid_f(to_f(gate[d + 1])) : y);
      }
    }
  }
}

// fp32 multiply-adds: 16 queries of a head and at most 8 VPT value columns per CTA; eight threads share a query.
constexpr int kVQ = 16, kVK = 32;

template <typename T, int VPT>
__global__ void __launch_bounds__(128) talk_values_kernel(const nb_talk_attention_args p, TalkBlock blk, int vtiles) {
  extern __shared__ __align__(16) float vsm[];   // [kVK][vn + 1] values, then [kVQ][kVK + 1] weights
  const int tid = threadIdx.x, qi = tid >> 3, sub = tid & 7;
  const int h = blockIdx.y / vtiles, v0 = (blockIdx.y - h * vtiles) * 8 * VPT, vn = min(8 * VPT, p.vdim - v0), b = blockIdx.z;
  const int local = blockIdx.x >> 2, r0 = (blockIdx.x & 3) * kVQ, q0 = (blk.tile0 + local) * kQT;
  if (q0 + r0 >= p.T) return;
  const int first = talk_first_key(p.pos0, q0, p.window), last = p.pos0 + min(q0 + kQT - 1, p.T - 1);
  const T* vals = reinterpret_cast<const T*>(p.cache) + (size_t)b * p.ctx * p.ldc + p.v_off + (h / (p.H / p.G)) * p.vdim + v0;
  const float* ws = blk.ws + (((size_t)(b * blk.tiles + local) * p.H + h) * kQT + r0 + qi) * blk.ld;
  float* p_s = vsm + kVK * (vn + 1);
  float m = -INFINITY, l = 0.f, acc[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) acc[i] = 0.f;
  for (int kc = first; kc <= last; kc += kVK) {
    __syncthreads();                     // the values before are no longer read
    for (int i = tid; i < kVK * vn; i += 128) {
      const int j = i / vn, d = i - j * vn;
      vsm[j * (vn + 1) + d] = kc + j <= last ? to_f(vals[(size_t)(kc + j) * p.ldc + d]) : 0.f;
    }
    float sc[4], cm = -INFINITY;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      sc[i] = ws[kc - first + sub + 8 * i];
      cm = fmaxf(cm, sc[i]);
    }
#pragma unroll
    for (int o = 1; o < 8; o <<= 1) cm = fmaxf(cm, __shfl_xor_sync(0xffffffffu, cm, o));
    const float m_new = fmaxf(m, cm), base = m_new == -INFINITY ? 0.f : m_new, corr = expf(m - base);
    float ps = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float e = expf(sc[i] - base);
      p_s[qi * (kVK + 1) + sub + 8 * i] = e;
      ps += e;
    }
#pragma unroll
    for (int o = 1; o < 8; o <<= 1) ps += __shfl_xor_sync(0xffffffffu, ps, o);
    l = l * corr + ps;
    m = m_new;
#pragma unroll
    for (int i = 0; i < VPT; ++i) acc[i] *= corr;
    __syncthreads();
    for (int j = 0; j < kVK; ++j) {
      const float w = p_s[qi * (kVK + 1) + j];
#pragma unroll
      for (int i = 0; i < VPT; ++i)
        if (sub + 8 * i < vn) acc[i] = fmaf(w, vsm[j * (vn + 1) + sub + 8 * i], acc[i]);
    }
  }
  if (q0 + r0 + qi < p.T) {
    const size_t row = (size_t)b * p.T + q0 + r0 + qi;
    const T* gate = p.gate ? reinterpret_cast<const T*>(p.gate) + row * p.ldg + h * p.vdim + v0 : nullptr;
    T* out = reinterpret_cast<T*>(p.out) + row * p.ldo + h * p.vdim + v0;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int d = sub + 8 * i;
      if (d < vn) out[d] = from_f<T>(acc[i] / l * (gate ? sigmoid_f(to_f(gate[d])) : 1.f));
    }
  }
}

// ---- one position per sequence.  grid (1, B, S) in clusters of S CTAs along z: a CTA takes a contiguous range of the
// window's keys for all heads (the heads of a key are mixed there), `stage` of them at a time from shared memory, with a
// running maximum and sum per head; then every CTA sends its weighted values in slices to the CTAs that merge them.  Rows
// of earlier positions, the talk matrix and the penalties do not depend on the launch before: they are requested ahead of
// the dependency wait.
constexpr int kTdThreads = 640, kTdWarps = kTdThreads / 32;

__host__ __device__ inline int pad4(int n) { return (n + 3) & ~3; }
// row length of a table [key][head]: a multiple of 4 that is odd in units of 4, so that 16-byte reads of neighbouring keys
// meet no bank twice
__host__ __device__ inline int head_row(int H) { return pad4(H) | 4; }

struct TalkDecodeSmem {                  // float offsets; the staged rows follow at `rows`
  int q, talk, sc, mx, acc, ml, xch, xml, wr, rows, dimp, hp, per, slot;
  __host__ __device__ TalkDecodeSmem(const nb_talk_decode_args& a, int S, int stage) {
    dimp = ((a.dim + 15) & ~15) + 8;     // rows of neighbouring heads start in different banks
    hp = head_row(a.H);
    per = pad4((a.H * a.vdim + S - 1) / S);
    slot = per;
    q = 0;
    talk = q + a.H * dimp;
    sc = talk + a.H * hp;
    mx = sc + stage * hp;
    acc = mx + stage * hp;
    ml = acc + pad4(a.H * a.vdim);
    xch = ml + 2 * hp;
    xml = xch + S * slot;
    wr = xml + S * 2 * hp;
    rows = wr + (S + 1) * hp;
  }
};

// i / n for small non-negative numbers
__device__ __forceinline__ int small_div(int i, int n) { return (int)__fdividef((float)i + 0.5f, (float)n); }

template <typename T> __device__ __forceinline__ int row_pad(int ldc) {      // 16-byte units of a staged row: odd
  return (ldc * (int)sizeof(T) / 16) | 1;
}

__device__ __forceinline__ void load8(const bf16* p, float (&v)[8]) {
  const uint4 t = *reinterpret_cast<const uint4*>(p);
  v[0] = bf_lo(t.x); v[1] = bf_hi(t.x); v[2] = bf_lo(t.y); v[3] = bf_hi(t.y);
  v[4] = bf_lo(t.z); v[5] = bf_hi(t.z); v[6] = bf_lo(t.w); v[7] = bf_hi(t.w);
}
__device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ float2 load2(const bf16* p) {
  const uint32_t t = *reinterpret_cast<const uint32_t*>(p);
  return make_float2(bf_lo(t), bf_hi(t));
}
__device__ __forceinline__ float2 load2(const float* p) { return *reinterpret_cast<const float2*>(p); }

template <typename T>
__global__ void __launch_bounds__(kTdThreads, 1) talk_decode_kernel(const nb_talk_decode_args p, int stage) {
  extern __shared__ __align__(16) float dsm[];
  cg::cluster_group cluster = cg::this_cluster();
  const int S = (int)cluster.num_blocks(), rank = (int)cluster.block_rank();
  const int b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const TalkDecodeSmem L(p, S, stage);
  const int H = p.H, rep = p.H / p.G, D = p.dim, V = p.vdim, hp = L.hp;
  float *qs = dsm + L.q, *talk_s = dsm + L.talk, *sc = dsm + L.sc, *mx = dsm + L.mx, *acc = dsm + L.acc, *ml = dsm + L.ml;
  float *xch = dsm + L.xch, *xml = dsm + L.xml, *wr = dsm + L.wr;
  T* rows = reinterpret_cast<T*>(dsm + L.rows);
  const int ldr16 = row_pad<T>(p.ldc);
  constexpr int kPiece = 16 / sizeof(T);
  const int ldr = ldr16 * kPiece, pieces = p.ldc / kPiece;

  const long long pos = *p.pos;          // written at the end of the step before
  if (pos < 0 || pos >= p.ctx) return;   // the same for every CTA
  const int n = p.window > 0 ? min((int)pos + 1, p.window) : (int)pos + 1, first = (int)pos + 1 - n;
  const int per = (n + S - 1) / S, k0 = first + rank * per, cnt = max(0, min(first + n, k0 + per) - k0);
  const int mine = (int)pos - k0;        // this position's place among this CTA's keys, if 0 <= mine < cnt
  T* cache = reinterpret_cast<T*>(p.cache) + (size_t)b * p.ctx * p.ldc;
  auto request = [&](int base, int m) {  // rows of earlier positions
    for (int j = warp; j < m; j += kTdWarps) {
      if (base + j == mine) continue;
      const T* src = cache + (size_t)(k0 + base + j) * p.ldc;
      T* dst = rows + (size_t)j * ldr;
      for (int c = lane; c < pieces; c += 32) cp16(dst + c * kPiece, src + c * kPiece);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto penalties = [&](int base, int m) {
    for (int i = tid; i < m * H; i += kTdThreads) {
      const int h = i / m, j = i - h * m;
      sc[j * hp + h] = p.penalty ? p.penalty[(size_t)h * p.n_pen + (int)pos - (k0 + base + j)] : 0.f;
    }
  };
  request(0, min(stage, cnt));
  for (int i = tid; i < H * hp; i += kTdThreads) {
    const int h = i / hp, g = i - h * hp;
    talk_s[i] = g < H ? p.talk[h * H + g] : 0.f;
  }
  for (int i = tid; i < stage * (hp - H); i += kTdThreads) {       // columns past the heads: read in fours
    const int j = i / (hp - H), c = H + i - j * (hp - H);
    sc[j * hp + c] = mx[j * hp + c] = 0.f;
  }
  penalties(0, min(stage, cnt));
  for (int i = tid; i < pad4(H * V); i += kTdThreads) acc[i] = 0.f;
  for (int i = tid; i < hp; i += kTdThreads) { ml[i] = -FLT_MAX; ml[hp + i] = 0.f; }
  cluster.barrier_arrive();

  pdl_enter();
  const float* row = p.p + (size_t)b * p.ldp;
  auto row_value = [&](int i) {          // element i of this position's row
    const bool in = i < p.G * D || (i >= p.v_off && i < p.v_off + p.G * V);
    return in ? row[p.k_off + i] : 0.f;
  };
  constexpr int kRowPre = 4;             // elements of it per thread that are requested with the queries
  float rv[kRowPre];
  if (mine >= 0 && mine < cnt) {
#pragma unroll
    for (int u = 0; u < kRowPre; ++u) rv[u] = tid + u * kTdThreads < p.ldc ? row_value(tid + u * kTdThreads) : 0.f;
  }
#pragma unroll 4
  for (int h = warp; h < H; h += kTdWarps)
#pragma unroll 4
    for (int d = lane; d < L.dimp; d += 32) qs[h * L.dimp + d] = d < D ? row[p.q_off + h * D + d] : 0.f;
  auto put_row = [&](T* dst) {           // this position's keys and values: staged, and into the cache
    T* crow = cache + (size_t)pos * p.ldc;
    auto put = [&](int i, float x) {
      const T v = from_f<T>(x);
      dst[i] = v;
      crow[i] = v;
    };
#pragma unroll
    for (int u = 0; u < kRowPre; ++u)
      if (tid + u * kTdThreads < p.ldc) put(tid + u * kTdThreads, rv[u]);
    for (int i = tid + kRowPre * kTdThreads; i < p.ldc; i += kTdThreads) put(i, row_value(i));
  };
  const bool dvec = D % 8 == 0, vvec = V % 2 == 0, mma = sizeof(T) == 2 && D % 8 == 0 && V % 8 == 0;
  const float isc = p.softcap > 0.f ? p.scale / p.softcap : p.scale;
  for (int base = 0; base < cnt; base += stage) {
    const int nk = min(stage, cnt - base);
    if (base > 0) {
      __syncthreads();                   // the rows and weights before are no longer read
      request(base, nk);
      penalties(base, nk);
    }
    if (mine >= base && mine < base + nk) put_row(rows + (size_t)(mine - base) * ldr);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const int chunks = (rep + 3) / 4, tiles8 = (rep + 7) / 8;
    auto put_score = [&](int j, int h, float x) {                  // over the penalty that waits there
      float* s = sc + j * hp + h;
      *s = (p.softcap > 0.f ? p.softcap * tanhf(x * isc) : x * isc) - *s;
    };
    const int ra = lane >> 2, c2 = (lane & 3) * 2;                 // of a product's fragments: this lane's row, its column pair
    if (mma) {
      // raw scores on the tensor cores: 16 keys x up to eight heads of a group per warp; the queries enter as three bf16
      // terms (a score's error is an exponent's)
      const int kt = (nk + 15) >> 4;
      for (int i = warp; i < p.G * tiles8 * kt; i += kTdWarps) {
        const int gc = small_div(i, kt), j0 = (i - gc * kt) * 16, g = small_div(gc, tiles8), hb = g * rep + (gc - g * tiles8) * 8;
        const int hn = min(8, (g + 1) * rep - hb);
        const bf16* kr = reinterpret_cast<const bf16*>(rows) + (size_t)min(j0 + (lane & 15), nk - 1) * ldr + g * D + (lane >> 4) * 8;
        const float* qr = qs + (hb + min(ra, hn - 1)) * L.dimp + c2;               // heads past the group's: not kept
        float c[3][4] = {};              // a chain of products per term
#pragma unroll 4
        for (int kk = 0; kk < D; kk += 16) {
          uint32_t a[4], q1[2], q2[2], q3[2];
          ldsm_x4(a, kr + kk);
#pragma unroll
          for (int f = 0; f < 2; ++f) {
            const float2 v = *reinterpret_cast<const float2*>(qr + kk + f * 8);
            split_bf16(v.x, v.y, q1[f], q2[f]);
            q3[f] = pack_bf16(v.x - bf_lo(q1[f]) - bf_lo(q2[f]), v.y - bf_hi(q1[f]) - bf_hi(q2[f]));
          }
          mma_bf16(c[0], a, q1[0], q1[1]);
          mma_bf16(c[1], a, q2[0], q2[1]);
          mma_bf16(c[2], a, q3[0], q3[1]);
        }
        float v[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float x = ((c[2][e] + c[1][e]) + c[0][e]) * isc;
          // cap tanh(x) = cap - 2 cap / (1 + e^2x): an absolute error of the cap's rounding
          v[e] = p.softcap > 0.f ? p.softcap - 2.f * p.softcap / (1.f + expf(2.f * x)) : x;
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int j = j0 + ra + (e >> 1) * 8, h = c2 + (e & 1);
          if (j < nk && h < hn) sc[j * hp + hb + h] = v[e] - sc[j * hp + hb + h];
        }
      }
    } else {
      // a thread takes one key of one group (and up to four of its heads at a time)
      for (int i = tid; i < nk * p.G * chunks; i += kTdThreads) {
        const int gc = small_div(i, nk), j = i - gc * nk, g = small_div(gc, chunks), h0 = g * rep + (gc - g * chunks) * 4, hn = min(4, (g + 1) * rep - h0);
        const T* kr = rows + (size_t)j * ldr + g * D;
        const float* qh = qs + h0 * L.dimp;
        float x[4] = {0.f, 0.f, 0.f, 0.f};
        if (dvec) {
          for (int d = 0; d < D; d += 8) {
            float kv[8];
            load8(kr + d, kv);
#pragma unroll
            for (int r = 0; r < 4; ++r)
              if (r < hn) {
                const float4 a = *reinterpret_cast<const float4*>(qh + r * L.dimp + d), c = *reinterpret_cast<const float4*>(qh + r * L.dimp + d + 4);
                x[r] += (kv[0] * a.x + kv[1] * a.y) + (kv[2] * a.z + kv[3] * a.w) + ((kv[4] * c.x + kv[5] * c.y) + (kv[6] * c.z + kv[7] * c.w));
              }
          }
        } else {
          for (int d = 0; d < D; ++d) {
            const float kv = to_f(kr[d]);
#pragma unroll
            for (int r = 0; r < 4; ++r)
              if (r < hn) x[r] = fmaf(kv, qh[r * L.dimp + d], x[r]);
          }
        }
#pragma unroll
        for (int r = 0; r < 4; ++r)
          if (r < hn) put_score(j, h0 + r, x[r]);
      }
    }
    __syncthreads();
    // mixed scores and the running softmax, a warp per head
    for (int h = warp; h < H; h += kTdWarps) {
      const float *t = talk_s + h * hp, old = ml[h];
      float m = old;
      for (int j = lane; j < nk; j += 64) {
        const bool two = j + 32 < nk;
        const float *s = sc + j * hp, *s2 = s + (two ? 32 * hp : 0);
        float v = 0.f, v2 = 0.f;
#pragma unroll 4
        for (int g = 0; g < hp; g += 4) {
          const float4 a = *reinterpret_cast<const float4*>(t + g), c = *reinterpret_cast<const float4*>(s + g);
          const float4 d = *reinterpret_cast<const float4*>(s2 + g);
          v += (a.x * c.x + a.y * c.y) + (a.z * c.z + a.w * c.w);
          v2 += (a.x * d.x + a.y * d.y) + (a.z * d.z + a.w * d.w);
        }
        mx[j * hp + h] = v;
        if (two) mx[(j + 32) * hp + h] = v2;
        m = fmaxf(m, fmaxf(v, v2));
      }
      m = warp_max(m);
      float sum = 0.f;
      for (int j = lane; j < nk; j += 32) {
        const float e = expf(mx[j * hp + h] - m);
        mx[j * hp + h] = e;
        sum += e;
      }
      sum = warp_sum(sum);
      if (lane == 0) {
        const float corr = expf(old - m);
        ml[h] = m;
        ml[hp + h] = ml[hp + h] * corr + sum;
        wr[h] = corr;
      }
    }
    __syncthreads();
    if (mma) {
      // weighted values: up to kCt tiles of 16 columns x up to eight heads of a group per warp; the weights enter as two bf16
      // terms
      constexpr int kCt = 4;
      const int ct = (V + 15) >> 4, tpw = min(kCt, (p.G * tiles8 * ct + kTdWarps - 1) / kTdWarps), parts = small_div(ct + tpw - 1, tpw);
      for (int i = warp; i < p.G * tiles8 * parts; i += kTdWarps) {
        const int gc = small_div(i, parts), t0 = (i - gc * parts) * tpw, g = small_div(gc, tiles8), hb = g * rep + (gc - g * tiles8) * 8;
        const int hn = min(8, (g + 1) * rep - hb), tn = min(tpw, ct - t0);
        // the values' tile, transposed: columns are the product's rows, keys its depth
        const bf16* vr = reinterpret_cast<const bf16*>(rows) + p.v_off + g * V + t0 * 16 + ((lane >> 3) & 1) * 8;
        const float* w = mx + hb + min(ra, hn - 1);                                // heads past the group's: not kept
        float c[kCt][2][4] = {};         // a chain of products per term
#pragma unroll 2
        for (int kk = 0; kk < nk; kk += 16) {
          uint32_t hi[2], lo[2];
#pragma unroll
          for (int f = 0; f < 2; ++f) {
            const int j = kk + f * 8 + c2;                                         // keys past the stage have no weight
            split_bf16(j < nk ? w[j * hp] : 0.f, j + 1 < nk ? w[(j + 1) * hp] : 0.f, hi[f], lo[f]);
          }
          const bf16* vk = vr + (size_t)min(kk + (lane & 7) + ((lane >> 4) << 3), nk - 1) * ldr;
#pragma unroll
          for (int y = 0; y < kCt; ++y)
            if (y < tn) {
              uint32_t a[4];
              ldsm_x4_t(a, vk + y * 16);
              mma_bf16(c[y][0], a, hi[0], hi[1]);
              mma_bf16(c[y][1], a, lo[0], lo[1]);
            }
        }
#pragma unroll
        for (int y = 0; y < kCt; ++y)
          if (y < tn) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int v = (t0 + y) * 16 + ra + (e >> 1) * 8, h = c2 + (e & 1);
              if (v < V && h < hn) {
                float* a = acc + (hb + h) * V + v;
                *a = fmaf(*a, wr[hb + h], c[y][0][e] + c[y][1][e]);
              }
            }
          }
      }
    } else {
      // a thread takes two columns (one if their number is odd) of up to four heads of a group
      const int vw = vvec ? 2 : 1, cols = V / vw;
      for (int i = tid; i < p.G * chunks * cols; i += kTdThreads) {
        const int gc = i / cols, c = (i - gc * cols) * vw, g = gc / chunks, h0 = g * rep + (gc - g * chunks) * 4, hn = min(4, (g + 1) * rep - h0);
        const T* vr = rows + p.v_off + g * V + c;
        float2 o[4] = {};
        if (vvec) {
#pragma unroll 4
          for (int j = 0; j < nk; ++j) {
            const float2 v = load2(vr + (size_t)j * ldr);
#pragma unroll
            for (int r = 0; r < 4; ++r)
              if (r < hn) {
                const float w = mx[j * hp + h0 + r];
                o[r].x = fmaf(w, v.x, o[r].x);
                o[r].y = fmaf(w, v.y, o[r].y);
              }
          }
        } else {
          for (int j = 0; j < nk; ++j) {
            const float v = to_f(vr[(size_t)j * ldr]);
#pragma unroll
            for (int r = 0; r < 4; ++r)
              if (r < hn) o[r].x = fmaf(mx[j * hp + h0 + r], v, o[r].x);
          }
        }
#pragma unroll
        for (int r = 0; r < 4; ++r)
          if (r < hn) {
            float* a = acc + (h0 + r) * V + c;
            a[0] = a[0] * wr[h0 + r] + o[r].x;
            if (vvec) a[1] = a[1] * wr[h0 + r] + o[r].y;
          }
      }
    }
  }
  __syncthreads();
  cluster.barrier_wait();                // every CTA of the cluster runs: its shared memory may be written from here on
  const int HV = H * V;
  for (int to = warp; to < S; to += kTdWarps) {  // slices, maxima and sums in fours; acc is padded to them
    float4* x = reinterpret_cast<float4*>(cluster.map_shared_rank(xch, to) + rank * L.slot);
    const float4* a = reinterpret_cast<const float4*>(acc + to * L.per);
    for (int i = lane; i < min(L.per, HV - to * L.per + 3) / 4; i += 32) x[i] = a[i];
    float4* y = reinterpret_cast<float4*>(cluster.map_shared_rank(xml, to) + rank * 2 * hp);
    for (int i = lane; i < hp / 2; i += 32) y[i] = reinterpret_cast<const float4*>(ml)[i];
  }
  // the gate of this CTA's slice travels meanwhile
  const int s0 = rank * L.per, sn = max(0, min(L.per, HV - s0));
  constexpr int kPre = 4;
  float gate[kPre];
#pragma unroll
  for (int u = 0; u < kPre; ++u) {
    const int i = tid + u * kTdThreads;
    gate[u] = p.g_off >= 0 && i < sn ? row[p.g_off + s0 + i] : 0.f;
  }
  cluster.sync();                        // nobody touches another CTA's shared memory after this
  for (int h = warp; h < H; h += kTdWarps) {       // a CTA without keys has maximum -FLT_MAX and sum 0
    const float mr = lane < S ? xml[lane * 2 * hp + h] : -FLT_MAX, w = expf(mr - warp_max(mr));
    const float den = warp_sum(lane < S ? w * xml[lane * 2 * hp + hp + h] : 0.f);
    if (lane < S) wr[lane * hp + h] = w;
    if (lane == 0) wr[S * hp + h] = 1.f / den;
  }
  __syncthreads();
  for (int i = tid, u = 0; i < sn; i += kTdThreads, ++u) {
    const int h = (s0 + i) / V;
    float v = 0.f;
    for (int r = 0; r < S; ++r) v = fmaf(wr[r * hp + h], xch[r * L.slot + i], v);
    v *= wr[S * hp + h];
    if (p.g_off >= 0) v *= sigmoid_f(u == 0 ? gate[0] : u == 1 ? gate[1] : u == 2 ? gate[2] : u == 3 ? gate[3] : row[p.g_off + s0 + i]);
    p.out[(size_t)b * p.ldo + s0 + i] = v;
  }
}

// ---------------------------------------------------------------- host
static int talk_ld(int T, int pos0, int window) {      // longest span of a query tile, rounded up to key tiles
  long long span = (long long)pos0 + T;
  if (window > 0) span = std::min<long long>(span, (long long)window + std::min(T, kQT) - 1);
  return (int)((span + kKT - 1) / kKT * kKT);
}

constexpr size_t kTalkSmem = 220 * 1024;

static size_t talk_scores_smem(const nb_talk_attention_args& a, int HM, int NB, int stages) {
  const int dkp = ((a.dim + 15) & ~15) + 8, KW = 64 * NB;
  return (size_t)(a.H * kSq + stages * KW) * dkp * 2 + ((size_t)a.H * HM + (size_t)a.H * (kSq + KW)) * 4;
}

template <int HM, int NB, bool kTwo> static int launch_scores_mma(const nb_talk_attention_args& a, const TalkBlock& blk, int stages, cudaStream_t st) {
  static bool done[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!done[dev & 63]) {
    if (cudaError_t e = cudaFuncSetAttribute(talk_scores_bf16_kernel<HM, NB, kTwo>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kTalkSmem))
      return record_cuda_error(e);
    done[dev & 63] = true;
  }
  const int vec = a.dim % 8 == 0 && a.ldq % 8 == 0 && a.ldc % 8 == 0 && (uintptr_t)a.q % 16 == 0 && (uintptr_t)a.cache % 16 == 0;
  const int steps = (blk.ld + 64 * NB - 1) / (64 * NB), subs = blk.tiles * (kQT / kSq);
  const int chunk = std::max(1, std::min(steps, (int)((long long)steps * subs * a.B / (2 * sm_count()))));   // about two CTAs per SM, one after the other
  talk_scores_bf16_kernel<HM, NB, kTwo><<<dim3((steps + chunk - 1) / chunk, subs, a.B), kScThreads, talk_scores_smem(a, HM, NB, stages), st>>>(
      a, blk, (a.dim + 15) & ~15, chunk, stages, vec);
  return check_launch();
}

// Whether the tensor-core kernel takes the sizes; launches it if so (rc: its status).
template <int HM, int NB> static bool launch_scores_bf16(const nb_talk_attention_args& a, const TalkBlock& blk, cudaStream_t st, int& rc) {
  const int stages = talk_scores_smem(a, HM, NB, 3) <= kTalkSmem ? 3 : 2;
  if (a.H > HM || talk_scores_smem(a, HM, NB, stages) > kTalkSmem) return false;
  rc = (a.H / a.G) % 2 == 0 ? launch_scores_mma<HM, NB, true>(a, blk, stages, st) : launch_scores_mma<HM, NB, false>(a, blk, stages, st);
  return true;
}

template <typename T> static int launch_scores_simple(const nb_talk_attention_args& a, const TalkBlock& blk, cudaStream_t st) {
  const size_t smem = ((size_t)a.H * 256 + (size_t)a.H * a.H) * 4;
  static bool done[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!done[dev & 63]) {
    if (cudaError_t e = cudaFuncSetAttribute(talk_scores_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 210 * 1024)) return record_cuda_error(e);
    done[dev & 63] = true;
  }
  talk_scores_kernel<T><<<dim3(blk.ld / kSt, blk.tiles * (kQT / kSt), a.B), 256, smem, st>>>(a, blk);
  return check_launch();
}

template <int VD> static int launch_values_bf16(const nb_talk_attention_args& a, const TalkBlock& blk, cudaStream_t st) {
  constexpr int smem = 2 * kKT * (VD + 8) * 2;
  const int vtiles = (a.vdim + VD - 1) / VD;
  static bool done[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!done[dev & 63]) {
    if (cudaError_t e = cudaFuncSetAttribute(talk_values_bf16_kernel<VD>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem)) return record_cuda_error(e);
    done[dev & 63] = true;
  }
  const int vec = a.vdim % 8 == 0 && a.ldc % 8 == 0 && a.v_off % 8 == 0 && a.ldo % 2 == 0 && a.ldg % 2 == 0 && (uintptr_t)a.cache % 16 == 0 &&
                  (uintptr_t)a.out % 4 == 0 && (uintptr_t)a.gate % 4 == 0;
  talk_values_bf16_kernel<VD><<<dim3(a.H * vtiles, blk.tiles, a.B), kPvThreads, smem, st>>>(a, blk, vtiles, vec);
  return check_launch();
}

template <typename T, int VPT> static int launch_values_simple(const nb_talk_attention_args& a, const TalkBlock& blk, cudaStream_t st) {
  const int vtiles = (a.vdim + 8 * VPT - 1) / (8 * VPT);
  const size_t smem = ((size_t)kVK * (std::min(8 * VPT, a.vdim) + 1) + kVQ * (kVK + 1)) * 4;
  talk_values_kernel<T, VPT><<<dim3(blk.tiles * (kQT / kVQ), a.H * vtiles, a.B), 128, smem, st>>>(a, blk, vtiles);
  return check_launch();
}

}  // namespace nb

using namespace nb;

extern "C" int nb_cache_append(const void* src, int ld, int off, int cols, void* cache, int ldc, int dtype, int B, int T, int ctx, int pos0,
                               void* stream) {
  if (!src || !cache || B < 1 || T < 1 || cols < 1 || off < 0 || pos0 < 0 || ctx < 1 || (dtype != NB_BF16 && dtype != NB_F32)) return NB_ERR_ARG;
  const int whole = (cols + 7) & ~7;
  if (off + whole > ld || whole > ldc || pos0 + T > ctx) return NB_ERR_SHAPE;
  if ((uintptr_t)src % 16 || (uintptr_t)cache % 16 || off % 8 || ld % 8 || ldc % 8) return NB_ERR_ALIGN;
  if (int rc = check_device()) return rc;
  const int per = dtype == NB_F32 ? 4 : 8;
  const long long total = (long long)B * T * (whole / per);
  return launch_pdl(cache_append_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, (cudaStream_t)stream,
                    reinterpret_cast<const uint4*>(src), ld / per, off / per, whole / per, reinterpret_cast<uint4*>(cache), ldc / per, T, ctx, pos0, total);
}

extern "C" size_t nb_talk_attention_workspace_bytes(int B, int T, int H, int pos0, int window, int query_tiles) {
  if (B < 1 || T < 1 || H < 1 || pos0 < 0 || window < 0 || query_tiles < 1) return 0;
  return (size_t)B * std::min(query_tiles, (T + kQT - 1) / kQT) * H * kQT * talk_ld(T, pos0, window) * 4;
}

extern "C" int nb_talk_attention(const nb_talk_attention_args* a, void* workspace, size_t workspace_bytes, void* stream) {
  if (!a || !a->q || !a->cache || !a->out || !a->talk || a->B < 1 || a->T < 1 || a->H < 1 || a->G < 1 || a->dim < 1 || a->vdim < 1 || a->pos0 < 0 ||
      a->window < 0 || a->v_off < 0)
    return NB_ERR_ARG;
  if (a->dtype != NB_BF16 && a->dtype != NB_F32) return NB_ERR_ARG;
  if (a->H % a->G || a->pos0 + a->T > a->ctx || a->v_off < a->G * a->dim || a->v_off + a->G * a->vdim > a->ldc || a->ldq < a->H * a->dim ||
      a->ldo < a->H * a->vdim || (a->gate && a->ldg < a->H * a->vdim) || a->B > 65535)
    return NB_ERR_SHAPE;
  const int most = a->window > 0 ? std::min(a->window, a->ctx) : a->ctx;
  if (a->penalty && a->n_pen < most) return NB_ERR_SHAPE;
  if ((size_t)a->H * (256 + a->H) * 4 > 200 * 1024 || (long long)a->H * ((a->vdim + 127) / 128) > 65535) return NB_ERR_SHAPE;
  const size_t one = nb_talk_attention_workspace_bytes(a->B, a->T, a->H, a->pos0, a->window, 1);
  if (!workspace || workspace_bytes < one) return NB_ERR_WORKSPACE;
  if ((uintptr_t)workspace % 256) return NB_ERR_ALIGN;
  if (int rc = check_device()) return rc;
  cudaStream_t st = (cudaStream_t)stream;
  const int all = (a->T + kQT - 1) / kQT, fit = std::min<size_t>(std::min<size_t>(workspace_bytes / one, all), 16000 / a->B + 1);
  const int blocks = (all + fit - 1) / fit, per = (all + blocks - 1) / blocks;     // equal blocks
  for (int t = 0; t < all; t += per) {
    TalkBlock blk;
    blk.ws = reinterpret_cast<float*>(workspace);
    blk.tile0 = t;
    blk.tiles = std::min(per, all - t);
    blk.ld = talk_ld(a->T, a->pos0, a->window);
    int rc = NB_OK;
    if (a->dtype == NB_F32) {
      rc = launch_scores_simple<float>(*a, blk, st);
    } else {
      const bool taken = (blk.ld > 256 && launch_scores_bf16<10, 4>(*a, blk, st, rc)) || launch_scores_bf16<10, 2>(*a, blk, st, rc) ||
                         (blk.ld > 64 && launch_scores_bf16<20, 2>(*a, blk, st, rc)) || launch_scores_bf16<20, 1>(*a, blk, st, rc) ||
                         launch_scores_bf16<40, 1>(*a, blk, st, rc);
      if (!taken) rc = launch_scores_simple<bf16>(*a, blk, st);
    }
    if (rc) return rc;
    if (a->dtype == NB_BF16)
      rc = a->vdim <= 64    ? launch_values_bf16<64>(*a, blk, st)
           : a->vdim <= 96  ? launch_values_bf16<96>(*a, blk, st)
           : a->vdim <= 128 ? launch_values_bf16<128>(*a, blk, st)
           : a->vdim <= 192 ? launch_values_bf16<192>(*a, blk, st)
                            : launch_values_bf16<256>(*a, blk, st);
    else
      rc = a->vdim <= 64 ? launch_values_simple<float, 8>(*a, blk, st) : a->vdim <= 128 ? launch_values_simple<float, 16>(*a, blk, st)
                                                                                         : launch_values_simple<float, 32>(*a, blk, st);
    if (rc) return rc;
  }
  return NB_OK;
}

template <typename T> static int launch_talk_decode(const nb_talk_decode_args& a, cudaStream_t st) {
  constexpr size_t kMax = 220 * 1024;
  auto kernel = talk_decode_kernel<T>;
  static int widest[64] = {};            // largest cluster the device takes
  int dev = 0;
  cudaGetDevice(&dev);
  cudaLaunchConfig_t cfg = {};
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = attr[0].val.clusterDim.y = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.blockDim = dim3(kTdThreads);
  cfg.stream = st;
  cfg.attrs = attr;
  if (!widest[dev & 63]) {
    if (cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kMax)) return record_cuda_error(e);
    if (cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeNonPortableClusterSizeAllowed, 1)) return record_cuda_error(e);
    attr[0].val.clusterDim.z = 16;
    cfg.gridDim = dim3(1, 1, 16);
    cfg.dynamicSmemBytes = kMax;
    cfg.numAttrs = 1;
    int n = 0;
    widest[dev & 63] = cudaOccupancyMaxActiveClusters(&n, kernel, &cfg) == cudaSuccess && n > 0 ? 16 : 8;
    cudaGetLastError();
  }
  const int most = a.window > 0 ? std::min(a.window, a.ctx) : a.ctx;
  int S = 1;
  while (S < widest[dev & 63] && S * 8 < most && a.B * S * 2 <= 256) S *= 2;
  const size_t row = (size_t)((a.ldc * sizeof(T) / 16) | 1) * 16, per_key = row + (size_t)2 * head_row(a.H) * 4;
  const size_t fixed = (size_t)TalkDecodeSmem(a, S, 0).rows * 4 + 32;
  if (fixed + per_key > kMax) return NB_ERR_SHAPE;
  const int stage = (int)std::min<size_t>((most + S - 1) / S, (kMax - fixed) / per_key);
  attr[0].val.clusterDim.z = S;
  cfg.gridDim = dim3(1, a.B, S);
  cfg.dynamicSmemBytes = (size_t)TalkDecodeSmem(a, S, stage).rows * 4 + stage * row + 32;   // 16-column reads of the last row
  cfg.numAttrs = 2;
  return record_cuda_error(cudaLaunchKernelEx(&cfg, kernel, a, stage));
}

extern "C" int nb_talk_decode(const nb_talk_decode_args* a, void* stream) {
  if (!a || !a->p || !a->cache || !a->talk || !a->pos || !a->out || a->B < 1 || a->H < 1 || a->G < 1 || a->dim < 1 || a->vdim < 1 || a->ctx < 1 ||
      a->window < 0 || a->q_off < 0 || a->k_off < 0 || a->v_off < 0)
    return NB_ERR_ARG;
  if (a->cache_dtype != NB_BF16 && a->cache_dtype != NB_F32) return NB_ERR_ARG;
  if (a->H % a->G || a->v_off < a->G * a->dim || a->v_off + a->G * a->vdim > a->ldc || a->q_off + a->H * a->dim > a->ldp ||
      a->k_off + a->v_off + a->G * a->vdim > a->ldp || (a->g_off >= 0 && a->g_off + a->H * a->vdim > a->ldp) || a->ldo < a->H * a->vdim ||
      a->B > 65535)
    return NB_ERR_SHAPE;
  const int most = a->window > 0 ? std::min(a->window, a->ctx) : a->ctx;
  if (a->penalty && a->n_pen < most) return NB_ERR_SHAPE;
  if ((uintptr_t)a->cache % 16 || a->ldc % 8 || a->v_off % 8) return NB_ERR_ALIGN;
  if (int rc = check_device()) return rc;
  return a->cache_dtype == NB_F32 ? launch_talk_decode<float>(*a, (cudaStream_t)stream) : launch_talk_decode<bf16>(*a, (cudaStream_t)stream);
}
