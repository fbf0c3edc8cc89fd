// Attention in the absorbed form over a ring of latent rows (layout: latent_rows.cuh): every query row -- one head of
// one token -- scores a cache row by the dot product of two rows and sums the rows' latents.
//
// The heads share the keys, so a tile is (rows = heads x tokens) x 64 keys on the tensor cores: 16 or 32 query rows per
// CTA, the key range split over CTAs.  Every part leaves its unnormalised sum, its largest score and its sum of
// exponentials; who reads them merges (latent_merge_kernel, or the staging of the value product of a one-token step).
// Key tiles are copied two deep by cp.async; a tile is read twice, as keys and (its first rankp columns) as values.
#pragma once

#include "act.cuh"
#include "latent_rows.cuh"
#include "rowvec.cuh"
#include "window_attention.cuh"

namespace tb {

constexpr int kLaThreads = 256, kLaWarps = 8, kLaKeys = 64;

struct LatentAttnParams {
  LatentRow r;
  int n_rows, tokens;           // query rows, row = head * tokens + token
  int ring, window;             // window 0: none
  const int* pos;               // position of token 0
  const float* q;               // [n_rows, r.row]
  const __nv_bfloat16* cache;   // [ring, r.row]
  float scale;
  int n_splits;
  float* part;                  // [n_rows, n_splits, rankp], then [n_rows, n_splits, 2]
};

__host__ __device__ inline size_t latent_attn_smem(int mt, int row) {
  return static_cast<size_t>(16 * mt + 2 * kLaKeys) * (row + 8) * 2 + static_cast<size_t>(16 * mt) * (kLaKeys + 8) * 2 +
         sizeof(float) * (2 + 1) * kLaWarps * 16 * mt;
}

// MT: tiles of 16 query rows; NV: blocks of 16 value columns per warp (rankp <= 128 * NV)
template <int MT, int NV>
__global__ void __launch_bounds__(kLaThreads, 1) latent_attn_kernel(const LatentAttnParams a) {
  extern __shared__ __align__(16) __nv_bfloat16 lsm[];
  constexpr int M = 16 * MT;
  constexpr int KG = kLaWarps / MT;      // warps side by side over the keys of a tile
  constexpr int KW = kLaKeys / KG;       // keys per warp: 8 or 16
  constexpr int PP = kLaKeys + 8;
  pdl_launch_dependents();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int row = a.r.row, kp = row + 8;
  __nv_bfloat16* qs = lsm;                          // [M][kp]
  __nv_bfloat16* ks = qs + M * kp;                  // [2][kLaKeys][kp]
  __nv_bfloat16* ps = ks + 2 * kLaKeys * kp;        // [M][PP]
  float* s_mx = reinterpret_cast<float*>(ps + M * PP);  // [2][KG][M]
  float* s_l = s_mx + 2 * kLaWarps * M;             // [KG][M]
  pdl_wait();
  const int pos0 = *a.pos;
  const int r0 = blockIdx.y * M, r1 = min(r0 + M, a.n_rows);
  // tokens of this tile: a range if it lies in one head, else all
  const bool one = r0 / a.tokens == (r1 - 1) / a.tokens;
  const int t_lo = one ? r0 % a.tokens : 0, t_hi = one ? (r1 - 1) % a.tokens : a.tokens - 1;
  const int first = a.window > 0 ? max(0, pos0 + t_lo - a.window + 1) : 0, last = pos0 + t_hi + 1;
  const int tiles = (last - first + kLaKeys - 1) / kLaKeys, per = (tiles + a.n_splits - 1) / a.n_splits * kLaKeys;
  const int lo = first + static_cast<int>(blockIdx.x) * per, hi = min(lo + per, last);
  float* ml = a.part + static_cast<long long>(a.n_rows) * a.n_splits * a.r.rankp;
  if (lo >= hi) {  // uniform over the CTA
    for (int i = tid; i < r1 - r0; i += kLaThreads) {
      float* d = ml + (static_cast<long long>(r0 + i) * a.n_splits + blockIdx.x) * 2;
      d[0] = -INFINITY;
      d[1] = 0.f;
    }
    return;
  }

  auto load_keys = [&](int buf, int k0) {
    const int slot0 = k0 % a.ring;
    __nv_bfloat16* dst = ks + buf * kLaKeys * kp;
#pragma unroll 2
    for (int r = warp; r < kLaKeys; r += kLaWarps) {
      const bool ok = k0 + r < hi;
      const long long slot = ok ? slot0 + r - (slot0 + r >= a.ring ? a.ring : 0) : 0;
      const __nv_bfloat16* src = a.cache + slot * row;
      for (int c = lane * 8; c < row; c += 256) cp_async16(dst + r * kp + c, src + c, ok);
    }
    cp_async_commit();
  };
  load_keys(0, lo);
  for (int i = tid; i < M * (row / 8); i += kLaThreads) {
    const int r = i / (row / 8), c = i - r * (row / 8);
    uint4 u = make_uint4(0u, 0u, 0u, 0u);
    if (r0 + r < r1) {
      float f[8];
      act_ld8(a.q + static_cast<long long>(r0 + r) * row + c * 8, f);
      u = make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
    }
    *reinterpret_cast<uint4*>(qs + r * kp + c * 8) = u;
  }

  const int mt = warp % MT, kg = warp / MT;          // scores: this warp's rows and keys
  const int srow = mt * 16 + (lane >> 2);            // and + 8
  int qpos[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = r0 + srow + 8 * i;
    qpos[i] = r < r1 ? pos0 + r % a.tokens : -1;     // a row that is none sees nothing
  }
  const int win = a.window > 0 ? a.window : 0x7fffffff;
  const int n_vb = a.r.rankp / 16;
  float o[MT][NV * 2][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < NV * 2; ++j)
#pragma unroll
      for (int q = 0; q < 4; ++q) o[i][j][q] = 0.f;
  float m_run[MT][2], l_run[2] = {0.f, 0.f};         // maxima of all rows a thread sums values for
#pragma unroll
  for (int i = 0; i < MT; ++i) m_run[i][0] = m_run[i][1] = -INFINITY;

  int buf = 0;
  for (int k0 = lo; k0 < hi; k0 += kLaKeys, buf ^= 1) {
    cp_async_wait<0>();
    __syncthreads();  // this tile is here, and the other buffer, ps and s_mx[buf] are free
    if (k0 + kLaKeys < hi) load_keys(buf ^ 1, k0 + kLaKeys);
    const __nv_bfloat16* kt = ks + buf * kLaKeys * kp;
    float s[KW / 8][4];
#pragma unroll
    for (int i = 0; i < KW / 8; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) s[i][j] = 0.f;
#pragma unroll 2
    for (int kk = 0; kk < row; kk += 32) {
      uint32_t qa[2][4];
      ldmatrix_x4(qa[0], qs + (mt * 16 + (lane & 15)) * kp + kk + (lane >> 4) * 8);
      ldmatrix_x4(qa[1], qs + (mt * 16 + (lane & 15)) * kp + kk + 16 + (lane >> 4) * 8);
#pragma unroll
      for (int i = 0; i < KW / 8; ++i) {
        uint32_t kb[4];  // eight keys, four pieces of eight along the row
        ldmatrix_x4(kb, kt + (kg * KW + i * 8 + (lane & 7)) * kp + kk + (lane >> 3) * 8);
        const uint32_t b0[2] = {kb[0], kb[1]}, b1[2] = {kb[2], kb[3]};
        mma_bf16_16816(s[i], qa[0], b0);
        mma_bf16_16816(s[i], qa[1], b1);
      }
    }
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int i = 0; i < KW / 8; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int kpos = k0 + kg * KW + i * 8 + (lane & 3) * 2 + (j & 1), q = j >> 1;
        const bool ok = kpos < hi && kpos <= qpos[q] && qpos[q] - kpos < win;
        s[i][j] = ok ? s[i][j] * a.scale : -INFINITY;
        mx[q] = fmaxf(mx[q], s[i][j]);
      }
    float* mxs = s_mx + buf * kLaWarps * M;
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      mx[q] = fmaxf(mx[q], __shfl_xor_sync(0xffffffffu, mx[q], 1));
      mx[q] = fmaxf(mx[q], __shfl_xor_sync(0xffffffffu, mx[q], 2));
      if ((lane & 3) == 0) mxs[kg * M + srow + 8 * q] = mx[q];
    }
    __syncthreads();
    float corr[MT][2], msafe[MT][2];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        float m = m_run[i][q];
#pragma unroll
        for (int g = 0; g < KG; ++g) m = fmaxf(m, mxs[g * M + i * 16 + (lane >> 2) + 8 * q]);
        msafe[i][q] = m == -INFINITY ? 0.f : m;
        corr[i][q] = __expf(m_run[i][q] - msafe[i][q]);
        m_run[i][q] = m;
      }
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      const float ms = MT == 1 || mt == 0 ? msafe[0][q] : msafe[MT - 1][q];
      l_run[q] *= MT == 1 || mt == 0 ? corr[0][q] : corr[MT - 1][q];
#pragma unroll
      for (int i = 0; i < KW / 8; ++i) {
        const float e0 = __expf(s[i][2 * q] - ms), e1 = __expf(s[i][2 * q + 1] - ms);
        l_run[q] += e0 + e1;
        *reinterpret_cast<uint32_t*>(ps + (srow + 8 * q) * PP + kg * KW + i * 8 + (lane & 3) * 2) = pack_bf16x2(e0, e1);
      }
    }
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int j = 0; j < NV * 2; ++j)
#pragma unroll
        for (int q = 0; q < 4; ++q) o[i][j][q] *= corr[i][q >> 1];
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < kLaKeys; kk += 16) {
      uint32_t pa[MT][4];
#pragma unroll
      for (int i = 0; i < MT; ++i) ldmatrix_x4(pa[i], ps + (i * 16 + (lane & 15)) * PP + kk + (lane >> 4) * 8);
#pragma unroll
      for (int j = 0; j < NV; ++j) {
        const int vb = warp + kLaWarps * j;
        if (vb < n_vb) {  // uniform over the warp
          uint32_t bv[4];
          ldmatrix_x4_trans(bv, kt + (kk + (lane & 15)) * kp + vb * 16 + (lane >> 4) * 8);
          const uint32_t b0[2] = {bv[0], bv[1]}, b1[2] = {bv[2], bv[3]};
#pragma unroll
          for (int i = 0; i < MT; ++i) {
            mma_bf16_16816(o[i][2 * j], pa[i], b0);
            mma_bf16_16816(o[i][2 * j + 1], pa[i], b1);
          }
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      const int r = r0 + i * 16 + (lane >> 2) + 8 * q;
      if (r >= r1) continue;
      float* dst = a.part + (static_cast<long long>(r) * a.n_splits + blockIdx.x) * a.r.rankp + (lane & 3) * 2;
#pragma unroll
      for (int j = 0; j < NV; ++j) {
        const int vb = warp + kLaWarps * j;
        if (vb < n_vb) {
          *reinterpret_cast<float2*>(dst + vb * 16) = make_float2(o[i][2 * j][2 * q], o[i][2 * j][2 * q + 1]);
          *reinterpret_cast<float2*>(dst + vb * 16 + 8) = make_float2(o[i][2 * j + 1][2 * q], o[i][2 * j + 1][2 * q + 1]);
        }
      }
    }
#pragma unroll
  for (int q = 0; q < 2; ++q) {
    l_run[q] += __shfl_xor_sync(0xffffffffu, l_run[q], 1);
    l_run[q] += __shfl_xor_sync(0xffffffffu, l_run[q], 2);
    if ((lane & 3) == 0) s_l[kg * M + srow + 8 * q] = l_run[q];
  }
  __syncthreads();
  // a warp's m_run covers every row; warp 0 writes the rows' maxima and sums
  if (warp == 0 && (lane & 3) == 0) {
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        const int lr = i * 16 + (lane >> 2) + 8 * q;
        if (r0 + lr >= r1) continue;
        float l = 0.f;
#pragma unroll
        for (int g = 0; g < KG; ++g) l += s_l[g * M + lr];
        float* d = ml + (static_cast<long long>(r0 + lr) * a.n_splits + blockIdx.x) * 2;
        d[0] = m_run[i][q];
        d[1] = l;
      }
  }
}

// ------------------------------------------------------------------ one-token products around it
// W_uk^T on the unrotated query, head by head (a block-diagonal product), the rotated query beside it, and the cache row
// of the token.
struct RvAbsorbParams {
  LatentRow r;
  Rotation rope;
  const float* q;           // per head ldh elements: dim unrotated, at dimp8 the part to rotate
  int heads, dim, dimp8, ldh;
  const __nv_bfloat16* w;   // [heads][rank][ldw]
  long long ldw;
  const float* c;           // [rank] latent
  const float* kr;          // [rot] key part
  const float* c_gain;
  float eps;
  const int* pos;
  int ring;
  float* lat;               // [heads][r.row]
  void* cache;
};

// Rows of a [heads][n][ldw] weight in groups of four rows of one head.
struct RvHeadsSrc {
  const __nv_bfloat16* w;
  long long ldw;
  int g0, gph, n;           // first group, groups per head, rows per head
  __device__ __forceinline__ uint4 load(int row, int piece) const {
    const int g = g0 + (row >> 2), h = g / gph, i = (g - h * gph) * 4 + (row & 3);
    return i < n ? ld_stream(w + (static_cast<long long>(h) * n + i) * ldw + piece * 8) : make_uint4(0u, 0u, 0u, 0u);
  }
};
struct RvHeadsVec {
  float* base;
  int stride, half;         // floats per vector, floats to the upper half
  int g0, gph, h0;
  __device__ __forceinline__ RvVec operator()(int group) const {
    float* p = base + ((g0 + group) / gph - h0) * stride;
    return {p, p + half};
  }
};

// Work split of a product head by head: CTA b has groups [g0, g1) of heads h0 .. h1.
struct RvHeadsRange {
  int gph, g0, g1, h0, h1;
  __host__ __device__ RvHeadsRange(int heads, int n, int b, int ctas) {
    gph = (n + 3) / 4;
    const long long groups = static_cast<long long>(heads) * gph;
    g0 = static_cast<int>(groups * b / ctas);
    g1 = static_cast<int>(groups * (b + 1) / ctas);
    h0 = g0 / gph;
    h1 = g1 > g0 ? (g1 - 1) / gph : h0;
  }
};
__host__ inline int rv_heads_span(int heads, int n, int ctas) {
  const int gph = (n + 3) / 4;
  const int span = (heads * gph + ctas - 1) / ctas / gph + 2;
  return span < heads ? span : heads;
}
__host__ __device__ inline int rv_vec_stride(int kp) { return rv_half_words(kp) + pad_to(kp / 2, 4); }

template <class Stage, class Emit>
__device__ __forceinline__ void rv_heads(const RvHeadsRange& rg, const __nv_bfloat16* w, long long ldw, int n, int k, float* smem,
                                         Stage stage, Emit emit) {
  const int kp = pad_to(k, 8);
  float* part = smem;
  float* vecs = smem + kRvBatchRows * kRvWarps;
  const RvTeam team(kp / 8);
  constexpr int kGroups = kRvBatchRows / kRvRows;
  uint4 ahead[kRvAhead + 1][kRvRows];
  {
    const RvHeadsSrc src{w, ldw, rg.g0, rg.gph, n};
    RvCursor c(team);
#pragma unroll
    for (int d = 0; d <= kRvAhead; ++d) {
      rv_load(src, team, c, min(rg.g1 - rg.g0, kGroups) * kRvRows, ahead[d]);
      c.next(team);
    }
  }
  pdl_wait();
  stage(vecs, rv_vec_stride(kp), rv_half_words(kp));
  __syncthreads();
  for (int b = rg.g0; b < rg.g1; b += kGroups) {
    const int rows = min(rg.g1 - b, kGroups) * kRvRows;
    rv_rows(RvHeadsSrc{w, ldw, b, rg.gph, n}, team, rows, RvHeadsVec{vecs, rv_vec_stride(kp), rv_half_words(kp), b, rg.gph, rg.h0}, part,
            ahead, b == rg.g0);
    __syncthreads();
    for (int i = threadIdx.x; i < rows; i += kRvThreads) {
      const int g = b + (i >> 2), h = g / rg.gph, e = (g - h * rg.gph) * 4 + (i & 3);
      if (e < n) emit(h, e, rv_total(team, part, i));
    }
    __syncthreads();
  }
}

template <typename T>
__global__ void __launch_bounds__(kRvThreads, 1) rv_absorb_kernel(const RvAbsorbParams p) {
  extern __shared__ __align__(16) float smem[];
  __shared__ float red[32];
  pdl_launch_dependents();
  const RvHeadsRange rg(p.heads, p.r.rank, blockIdx.x, gridDim.x);
  auto stage = [&](float* vecs, int stride, int half) {
    const int per = p.dimp8 / 4;
    for (int i = threadIdx.x; i < (rg.h1 - rg.h0 + 1) * per; i += kRvThreads) {
      const int h = i / per, g = i - h * per;
      const RvVec v{vecs + h * stride, vecs + h * stride + half};
      v.put4(g, reinterpret_cast<const float4*>(p.q + static_cast<long long>(rg.h0 + h) * p.ldh)[g]);
    }
  };
  auto emit = [&](int h, int e, float v) { p.lat[static_cast<long long>(h) * p.r.row + e] = v; };
  rv_heads(rg, p.w, p.ldw, p.r.rank, p.dim, smem, stage, emit);
  const int pos = *p.pos;
  for (int h = blockIdx.x; h < p.heads; h += gridDim.x) {
    const float* src = p.q + static_cast<long long>(h) * p.ldh + p.dimp8;
    for (int e = threadIdx.x; e < p.r.rot; e += kRvThreads)
      p.lat[static_cast<long long>(h) * p.r.row + p.r.rankp + e] = p.rope(pos, e, [&](int i) { return src[i]; });
  }
  if (blockIdx.x == gridDim.x - 1) {
    float sc = 0.f;
    for (int i = threadIdx.x; i < p.r.rank; i += kRvThreads) sc += p.c[i] * p.c[i];
    const float rc = 1.f / sqrtf(cta_sum(sc, red) / static_cast<float>(p.r.rank) + p.eps);
    T* dst = reinterpret_cast<T*>(p.cache) + static_cast<long long>(pos % p.ring) * p.r.row;
    for (int i = threadIdx.x; i < p.r.rank; i += kRvThreads) act_st(dst + i, p.c[i] * rc * p.c_gain[i]);
    for (int e = threadIdx.x; e < p.r.rot; e += kRvThreads) act_st(dst + p.r.rankp + e, p.rope(pos, e, [&](int i) { return p.kr[i]; }));
  }
}

// The value expansion of one token, head by head, on the merged parts of its attention; the output gate on top.
struct RvValueParams {
  LatentRow r;
  const float* part;        // [heads, n_splits, rankp], then [heads, n_splits, 2]
  int heads, vdim, n_splits;
  const float* sink;        // optional [heads]
  const __nv_bfloat16* w;   // [heads][vdim][ldw]
  long long ldw;
  HeadGate gate;
  float* out;               // [heads * vdim]
};

static __global__ void __launch_bounds__(kRvThreads, 1) rv_value_kernel(const RvValueParams p) {
  extern __shared__ __align__(16) float smem[];
  pdl_launch_dependents();
  const RvHeadsRange rg(p.heads, p.vdim, blockIdx.x, gridDim.x);
  const int span = rg.h1 - rg.h0 + 1, rp8 = pad_to(p.r.rank, 8);
  auto stage = [&](float* vecs, int stride, int half) {
    float* wgt = vecs + span * stride;
    const float* ml = p.part + static_cast<long long>(p.heads) * p.n_splits * p.r.rankp;
    for (int h = threadIdx.x >> 5; h < span; h += kRvWarps)
      part_weights(ml + static_cast<long long>(rg.h0 + h) * p.n_splits * 2, p.n_splits, p.sink != nullptr ? p.sink + rg.h0 + h : nullptr,
                   wgt + h * p.n_splits);
    __syncthreads();
    for (int i = threadIdx.x; i < span * (rp8 / 4); i += kRvThreads) {
      const int h = i / (rp8 / 4), g = i - h * (rp8 / 4);
      const RvVec v{vecs + h * stride, vecs + h * stride + half};
      float4 o = merged4(p.part + static_cast<long long>(rg.h0 + h) * p.n_splits * p.r.rankp, wgt + h * p.n_splits, p.n_splits, p.r.rankp, g);
      v.put4(g, o);
    }
  };
  auto emit = [&](int h, int e, float v) { p.out[h * p.vdim + e] = v * p.gate(0, h, p.vdim, e); };
  rv_heads(rg, p.w, p.ldw, p.vdim, p.r.rank, smem, stage, emit);
}

}  // namespace tb
