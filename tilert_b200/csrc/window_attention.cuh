// Grouped-query attention over a ring of cached keys and values.
//
// A cache holds, per key/value head, `ring` rows; position p lives in row p mod ring.  A query at position i sees
// the positions j with 0 <= i - j < window (window 0: every j <= i); the ring has to hold the window of the oldest
// query of a launch together with every position of the launch.  Rows are padded to 16 elements with zeros.
//
// Queries and keys are RMS-normalised over their whole projection, one statistic for all heads; values can be blended
// with what an earlier layer computed at that position.  Both happen here:
//   qkv_rows_kernel          a portion of tokens: normalised queries out, keys and values into the ring
//   attn_prefill_kernel      a portion of tokens, bf16 tensor-core tiles with an online softmax
//   attn_rows_kernel<T, true>   one token: the preparation, the cache write and the attention in one launch, the
//                            keys split over CTAs, the last CTA of a head block merging the parts
//   attn_rows_kernel<T, false>  any number of prepared query rows, f32 arithmetic (the exact mode)
// The last two read keys and values through strides, so that values may lie inside the keys' rows (a latent cache) or
// keys may be two pieces, one of them shared by all heads.  The prefill kernel takes an optional sink per head (one more
// term of the softmax denominator, without key or value) and an optional output gate.
// Scores, softmax and sums are f32 throughout.
#pragma once

#include "act.cuh"

namespace tb {

enum ValueMix : int { VMIX_NONE = 0, VMIX_FIRST = 1, VMIX_BLEND = 2 };

struct QkvShape {
  int heads, kv_heads, dim, vdim;
  int dimp, vdimp;       // padded to 16
  int ring;              // cache rows per head
  int window;            // 0: no window
};

struct QkvPrep {
  const float* qkv;      // [rows, ld]: queries, keys, values of one token
  long long ld;
  const float* q_gain;   // [heads * dim]
  const float* k_gain;   // [kv_heads * dim]
  float eps;
  int v_mode;
  const float* lambda;   // one value (VMIX_BLEND)
  float* v_first;        // [rows, kv_heads * vdim] written (VMIX_FIRST) or read (VMIX_BLEND)
};

// Value element e (over all heads) of row `t`, after mixing; VMIX_FIRST also leaves it for the later layers.
__device__ __forceinline__ float mixed_value(const QkvPrep& p, const QkvShape& s, int t, int e, bool store_first) {
  const int nq = s.heads * s.dim, nk = s.kv_heads * s.dim, nv = s.kv_heads * s.vdim;
  const float v = p.qkv[t * p.ld + nq + nk + e];
  if (p.v_mode == VMIX_FIRST && store_first) p.v_first[static_cast<long long>(t) * nv + e] = v;
  if (p.v_mode == VMIX_BLEND) {
    const float l = *p.lambda;
    return (1.f - l) * v + l * p.v_first[static_cast<long long>(t) * nv + e];
  }
  return v;
}

// This thread's share of the sum of squares of row[0..n).
__device__ __forceinline__ float sum_squares(const float* row, int n) {
  float s = 0.f;
  if (n % 4 == 0 && reinterpret_cast<uintptr_t>(row) % 16 == 0) {
    const float4* r4 = reinterpret_cast<const float4*>(row);
#pragma unroll 4
    for (int i = threadIdx.x; i < n / 4; i += blockDim.x) {
      const float4 v = r4[i];
      s += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
    }
  } else {
    for (int i = threadIdx.x; i < n; i += blockDim.x) s += row[i] * row[i];
  }
  return s;
}

__device__ __forceinline__ float rinv_of(float sum, int n, float eps) { return 1.f / sqrtf(sum / static_cast<float>(n) + eps); }

// ------------------------------------------------------------------ a portion of tokens: prepare
struct QkvRowsParams {
  QkvShape s;
  QkvPrep p;
  const int* pos;        // position of row 0
  void* q;               // [rows, heads, dimp] normalised queries (padding left as it is: zero)
  void* k_cache;         // [kv_heads, ring, dimp]
  void* v_cache;         // [kv_heads, ring, vdimp]
};

template <typename T>
__global__ void __launch_bounds__(256) qkv_rows_kernel(const QkvRowsParams a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[32];
  const QkvShape& s = a.s;
  const int t = blockIdx.x;
  const float* row = a.p.qkv + t * a.p.ld;
  const int nq = s.heads * s.dim, nk = s.kv_heads * s.dim, nv = s.kv_heads * s.vdim;
  const float sq = sum_squares(row, nq), sk = sum_squares(row + nq, nk);
  const float rq = rinv_of(cta_sum(sq, red), nq, a.p.eps), rk = rinv_of(cta_sum(sk, red), nk, a.p.eps);
  const long long slot = (*a.pos + t) % s.ring;
  T* q = reinterpret_cast<T*>(a.q) + static_cast<long long>(t) * s.heads * s.dimp;
  T* kc = reinterpret_cast<T*>(a.k_cache);
  T* vc = reinterpret_cast<T*>(a.v_cache);
  for (int i = threadIdx.x; i < nq; i += 256) {
    const int h = i / s.dim;
    act_st(q + h * s.dimp + i - h * s.dim, row[i] * rq * a.p.q_gain[i]);
  }
  for (int i = threadIdx.x; i < nk; i += 256) {
    const int g = i / s.dim;
    act_st(kc + (static_cast<long long>(g) * s.ring + slot) * s.dimp + i - g * s.dim, row[nq + i] * rk * a.p.k_gain[i]);
  }
  for (int i = threadIdx.x; i < nv; i += 256) {
    const int g = i / s.vdim;
    act_st(vc + (static_cast<long long>(g) * s.ring + slot) * s.vdimp + i - g * s.vdim, mixed_value(a.p, s, t, i, true));
  }
}

// ------------------------------------------------------------------ query rows against a range of keys, f32
constexpr int kAttnThreads = 256;
constexpr int kAttnHeads = 4;    // query heads per CTA
constexpr int kAttnChunk = 128;  // keys per softmax step
constexpr int kAttnPasses = kAttnChunk / 32;
constexpr int kAttnAhead = 4;    // value rows a thread loads together
static_assert(kAttnThreads == 256, "eight warps of four keys make a pass of 32");

struct AttnRowsParams {
  QkvShape s;
  QkvPrep p;             // FUSED
  const int* pos;        // position of row 0
  const void* q;         // !FUSED: row of (head, token) at head * q_head + token * q_token, element type QT
  long long q_head, q_token;
  void* k_cache;
  void* v_cache;
  long long v_ld;        // elements between value rows
  int rows;
  int parts_only;        // leave every part (n_splits may be 1) for the caller to merge; `out` is not written
  float scale;
  int n_splits;
  float* part;           // [heads, rows, n_splits, vdimp] and, behind it, [heads, rows, n_splits, 2] (max, sum)
  unsigned* counter;     // [head blocks], zero between launches
  void* out;             // [rows, ldo], element type float (FUSED) or T
  long long ldo;
};

__host__ __device__ inline size_t attn_rows_smem(int dimp, int vdimp) {
  return (kAttnHeads * dimp + kAttnHeads * kAttnChunk + kAttnThreads * kAttnHeads * 8) * sizeof(float);
}

// Key range of one part of a query at `pos`.
struct KeyRange {
  int lo, hi;
};
__device__ __forceinline__ KeyRange key_range(int pos, int window, int n_splits, int split) {
  const int first = window > 0 ? max(0, pos - window + 1) : 0;
  const int per = (pos + 1 - first + n_splits - 1) / n_splits;
  const int lo = min(first + split * per, pos + 1);
  return {lo, min(lo + per, pos + 1)};
}

// Requests the part's cached rows into the L2 before the launch may read anything (a hint: what it reads of the
// position may be old, the addresses stay inside the cache either way).
template <typename T>
__device__ __forceinline__ void prefetch_range(const AttnRowsParams& a, int g) {
  const QkvShape& s = a.s;
  const KeyRange r = key_range(max(*reinterpret_cast<const volatile int*>(a.pos), 0), s.window, a.n_splits, blockIdx.x);
  for (int key = r.lo + static_cast<int>(threadIdx.x); key < r.hi; key += kAttnThreads) {
    const long long row = static_cast<long long>(g) * s.ring + key % s.ring;
    const char* k = reinterpret_cast<const char*>(reinterpret_cast<const T*>(a.k_cache) + row * s.dimp);
    const char* v = reinterpret_cast<const char*>(reinterpret_cast<const T*>(a.v_cache) + row * s.vdimp);
    for (int b = 0; b < s.dimp * static_cast<int>(sizeof(T)); b += 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(k + b));
    for (int b = 0; b < s.vdimp * static_cast<int>(sizeof(T)); b += 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(v + b));
  }
}

template <typename T, bool FUSED, typename QT = T>
__global__ void __launch_bounds__(kAttnThreads) attn_rows_kernel(const AttnRowsParams a) {
  extern __shared__ __align__(16) float smem[];
  __shared__ float red[32];
  __shared__ float s_m[kAttnHeads], s_l[kAttnHeads], s_corr[kAttnHeads];
  __shared__ int s_last;
  pdl_launch_dependents();
  const QkvShape& s = a.s;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (FUSED) prefetch_range<T>(a, blockIdx.y / ((s.heads / s.kv_heads + kAttnHeads - 1) / kAttnHeads));
  pdl_wait();
  const int group = s.heads / s.kv_heads, n_hb = (group + kAttnHeads - 1) / kAttnHeads;
  const int split = blockIdx.x, g = blockIdx.y / n_hb, hb = blockIdx.y - g * n_hb, t = blockIdx.z;
  const int h0 = g * group + hb * kAttnHeads;
  const int nh = min(kAttnHeads, group - hb * kAttnHeads);
  const int pos = *a.pos + t;
  float* qs = smem;                               // [kAttnHeads][dimp], scaled
  float* sc = qs + kAttnHeads * s.dimp;           // [kAttnHeads][kAttnChunk]
  float* red2 = sc + kAttnHeads * kAttnChunk;     // [threads][kAttnHeads * 8]
  const KeyRange range = key_range(pos, s.window, a.n_splits, split);
  const int lo = range.lo, hi = range.hi;
  T* kc = reinterpret_cast<T*>(a.k_cache) + static_cast<long long>(g) * s.ring * s.dimp;
  T* vc = reinterpret_cast<T*>(a.v_cache) + static_cast<long long>(g) * s.ring * a.v_ld;

  if (FUSED) {
    const int nq = s.heads * s.dim, nk = s.kv_heads * s.dim;
    const float* row = a.p.qkv;
    const float sq = sum_squares(row, nq), sk = sum_squares(row + nq, nk);
    const float rq = rinv_of(cta_sum(sq, red), nq, a.p.eps), rk = rinv_of(cta_sum(sk, red), nk, a.p.eps);
    for (int i = tid; i < kAttnHeads * s.dimp; i += kAttnThreads) {
      const int h = i / s.dimp, d = i - h * s.dimp;
      const int e = (h0 + h) * s.dim + d;
      qs[i] = h < nh && d < s.dim ? row[e] * rq * a.p.q_gain[e] * a.scale : 0.f;
    }
    if (lo < hi && hi == pos + 1) {  // the CTAs whose range holds the current position write (the same) cache row
      const long long slot = pos % s.ring;
      for (int d = tid; d < s.dim; d += kAttnThreads) {
        const int e = g * s.dim + d;
        act_st(kc + slot * s.dimp + d, row[nq + e] * rk * a.p.k_gain[e]);
      }
      for (int d = tid; d < s.vdim; d += kAttnThreads)
        act_st(vc + slot * a.v_ld + d, mixed_value(a.p, s, 0, g * s.vdim + d, true));
    }
  } else {
    const QT* q = reinterpret_cast<const QT*>(a.q) + t * a.q_token + h0 * a.q_head;
    for (int i = tid; i < kAttnHeads * s.dimp; i += kAttnThreads) {
      const int h = i / s.dimp;
      qs[i] = h < nh ? act_ld(q + h * a.q_head + (i - h * s.dimp)) * a.scale : 0.f;
    }
  }
  if (tid < kAttnHeads) {
    s_m[tid] = -INFINITY;
    s_l[tid] = 0.f;
  }
  __syncthreads();  // queries staged, the current cache row visible to this CTA

  const int n_vc = s.vdimp / 8;                    // value pieces; thread = (key lane, piece)
  const int key_lanes = kAttnThreads / n_vc;
  const int kl = tid / n_vc, vp = tid - kl * n_vc;
  const bool v_active = kl < key_lanes;
  float acc[kAttnHeads][8];
#pragma unroll
  for (int h = 0; h < kAttnHeads; ++h)
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[h][j] = 0.f;

  // the keys of a launch lie in fewer than `ring` consecutive positions, so one subtraction wraps a row index
  for (int c0 = lo; c0 < hi; c0 += kAttnChunk) {
    const int cn = min(kAttnChunk, hi - c0), slot0 = c0 % s.ring;
    // scores: eight lanes per key, four keys per warp and pass; the passes' keys are loaded together
    const int cn32 = pad_to(cn, 32);
    {
      const T* kr[kAttnPasses];
      float d[kAttnPasses][kAttnHeads];
#pragma unroll
      for (int it = 0; it < kAttnPasses; ++it) {
        const int key = min(it * 32 + warp * 4 + (lane >> 3), cn - 1);  // past the end: the last key, dropped below
        const int slot = slot0 + key - (slot0 + key >= s.ring ? s.ring : 0);
        kr[it] = kc + static_cast<long long>(slot) * s.dimp;
#pragma unroll
        for (int h = 0; h < kAttnHeads; ++h) d[it][h] = 0.f;
      }
#pragma unroll 2
      for (int c = lane & 7; c < s.dimp / 8; c += 8) {
        float f[kAttnPasses][8];
#pragma unroll
        for (int it = 0; it < kAttnPasses; ++it)
          if (it * 32 < cn) act_ld8(kr[it] + c * 8, f[it]);
#pragma unroll
        for (int h = 0; h < kAttnHeads; ++h) {
          const float4 q0 = *reinterpret_cast<const float4*>(qs + h * s.dimp + c * 8);
          const float4 q1 = *reinterpret_cast<const float4*>(qs + h * s.dimp + c * 8 + 4);
#pragma unroll
          for (int it = 0; it < kAttnPasses; ++it)
            if (it * 32 < cn)
              d[it][h] += f[it][0] * q0.x + f[it][1] * q0.y + f[it][2] * q0.z + f[it][3] * q0.w + f[it][4] * q1.x + f[it][5] * q1.y +
                          f[it][6] * q1.z + f[it][7] * q1.w;
        }
      }
#pragma unroll
      for (int it = 0; it < kAttnPasses; ++it)
        if (it * 32 < cn) {
          const int key = it * 32 + warp * 4 + (lane >> 3);
#pragma unroll
          for (int h = 0; h < kAttnHeads; ++h) {
#pragma unroll
            for (int o = 4; o > 0; o >>= 1) d[it][h] += __shfl_xor_sync(0xffffffffu, d[it][h], o);
            if ((lane & 7) == 0) sc[h * kAttnChunk + key] = key < cn ? d[it][h] : -INFINITY;
          }
        }
    }
    __syncthreads();
    if (warp < kAttnHeads) {
      float m = -INFINITY;
      for (int i = lane; i < cn32; i += 32) m = fmaxf(m, sc[warp * kAttnChunk + i]);
      m = fmaxf(warp_max(m), s_m[warp]);
      float l = 0.f;
      for (int i = lane; i < cn32; i += 32) {
        const float e = expf(sc[warp * kAttnChunk + i] - m);
        sc[warp * kAttnChunk + i] = e;
        l += e;
      }
      l = warp_sum(l);
      if (lane == 0) {
        const float corr = expf(s_m[warp] - m);
        s_corr[warp] = corr;
        s_l[warp] = s_l[warp] * corr + l;
        s_m[warp] = m;
      }
    }
    __syncthreads();
    if (v_active) {
#pragma unroll
      for (int h = 0; h < kAttnHeads; ++h)
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[h][j] *= s_corr[h];
      for (int k0 = kl; k0 < cn; k0 += kAttnAhead * key_lanes) {
        float f[kAttnAhead][8];
#pragma unroll
        for (int u = 0; u < kAttnAhead; ++u) {
          const int key = min(k0 + u * key_lanes, cn - 1);
          const int slot = slot0 + key - (slot0 + key >= s.ring ? s.ring : 0);
          act_ld8(vc + slot * a.v_ld + vp * 8, f[u]);
        }
#pragma unroll
        for (int u = 0; u < kAttnAhead; ++u) {
          const int key = k0 + u * key_lanes;
#pragma unroll
          for (int h = 0; h < kAttnHeads; ++h) {
            const float w = key < cn ? sc[h * kAttnChunk + key] : 0.f;
#pragma unroll
            for (int j = 0; j < 8; ++j) acc[h][j] += w * f[u][j];
          }
        }
      }
    }
    __syncthreads();
  }

  // sum over the key lanes: red2[kl][h][vdimp]
  if (v_active) {
#pragma unroll
    for (int h = 0; h < kAttnHeads; ++h)
#pragma unroll
      for (int j = 0; j < 8; ++j) red2[(kl * kAttnHeads + h) * s.vdimp + vp * 8 + j] = acc[h][j];
  }
  __syncthreads();
  const bool whole = a.n_splits == 1 && !a.parts_only;
  float* ml = a.part + static_cast<long long>(s.heads) * a.rows * a.n_splits * s.vdimp;
  auto part_of = [&](int h) { return (static_cast<long long>(h0 + h) * a.rows + t) * a.n_splits; };
  for (int i = tid; i < nh * s.vdimp; i += kAttnThreads) {
    const int h = i / s.vdimp, v = i - h * s.vdimp;
    float o = 0.f;
    for (int k = 0; k < key_lanes; ++k) o += red2[(k * kAttnHeads + h) * s.vdimp + v];
    if (!whole) {
      a.part[(part_of(h) + split) * s.vdimp + v] = o;
    } else if (v < s.vdim) {
      const long long dst = t * a.ldo + (h0 + h) * s.vdim + v;
      if (FUSED)
        reinterpret_cast<float*>(a.out)[dst] = o / s_l[h];
      else
        act_st(reinterpret_cast<T*>(a.out) + dst, o / s_l[h]);
    }
  }
  if (whole) return;
  if (tid < nh) {
    ml[(part_of(tid) + split) * 2] = s_m[tid];
    ml[(part_of(tid) + split) * 2 + 1] = s_l[tid];
  }
  if (a.parts_only) return;
  // merge by the CTA that finishes its head block last (no CTA waits for another)
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    const unsigned prev = atomicAdd(a.counter + blockIdx.y, 1u);
    s_last = prev == static_cast<unsigned>(a.n_splits) - 1u;
    if (s_last) a.counter[blockIdx.y] = 0u;
  }
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  // weight of every part, one warp per head: exp(max - overall max), and the overall sum (red2 is free again)
  float* wgt = red2;  // [kAttnHeads][n_splits]
  if (warp < nh) {
    const float* mh = ml + part_of(warp) * 2;
    float m = -INFINITY, l = 0.f;
    for (int k = lane; k < a.n_splits; k += 32) m = fmaxf(m, __ldcg(mh + 2 * k));
    m = warp_max(m);
    for (int k = lane; k < a.n_splits; k += 32) {
      const float c = expf(__ldcg(mh + 2 * k) - m);  // an empty part has max -inf: weight 0
      wgt[warp * a.n_splits + k] = c;
      l += c * __ldcg(mh + 2 * k + 1);
    }
    l = warp_sum(l);
    if (lane == 0) s_l[warp] = l;
  }
  __syncthreads();
  for (int i = tid; i < nh * s.vdim; i += kAttnThreads) {
    const int h = i / s.vdim, v = i - h * s.vdim;
    const float* src = a.part + part_of(h) * s.vdimp + v;
    const float* w = wgt + h * a.n_splits;
    float o = 0.f;
#pragma unroll 8
    for (int k = 0; k < a.n_splits; ++k) o += w[k] * __ldcg(src + static_cast<long long>(k) * s.vdimp);
    const long long dst = t * a.ldo + (h0 + h) * s.vdim + v;
    if (FUSED)
      reinterpret_cast<float*>(a.out)[dst] = o / s_l[h];
    else
      act_st(reinterpret_cast<T*>(a.out) + dst, o / s_l[h]);
  }
}

// ------------------------------------------------------------------ a portion of tokens, bf16 tensor-core tiles
// 64 rows per CTA = (tokens x query heads of one key/value head), so the heads of a group share the key tiles.
// 64 keys per tile; the next keys are requested (cp.async) before a tile's scores, the next values after its product;
// four warps of 16 rows, three CTAs per SM at 128-wide heads; online softmax in registers.
constexpr int kFaRows = 64, kFaKeys = 64, kFaThreads = 128;
constexpr int kFaMaxHeads = 16;  // query heads of a group per CTA

struct AttnPrefillParams {
  QkvShape s;
  const int* pos;        // position of row 0
  int rows;
  const __nv_bfloat16* q;        // [rows, heads, dimp]
  // A key row is dim1 elements of k_cache (head g, row r at g * k_head + r * k_ld), then dimp - dim1 of k2 (row r at
  // r * k2_ld, the same for all heads); a value row lies at g * v_head + r * v_ld.
  const __nv_bfloat16* k_cache;
  const __nv_bfloat16* k2;
  const __nv_bfloat16* v_cache;
  long long k_head, k_ld, k2_ld, v_head, v_ld;
  int dim1;
  float scale;
  const float* sink;     // optional [heads]
  HeadGate gate;         // of the output
  __nv_bfloat16* out;    // [rows, ldo]
  long long ldo;
};

__host__ __device__ inline size_t attn_prefill_smem(int dimp, int vdimp) {
  return (static_cast<size_t>(kFaRows + 2 * kFaKeys) * (dimp + 8) + kFaKeys * (vdimp + 8)) * 2;
}

__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// DV16: value tiles of 16 columns the accumulator has room for (vdimp <= 16 * DV16)
template <int DV16>
__global__ void __launch_bounds__(kFaThreads, DV16 <= 8 ? 3 : 1) attn_prefill_kernel(const AttnPrefillParams a) {
  extern __shared__ __align__(16) __nv_bfloat16 fsm[];
  pdl_launch_dependents();
  pdl_wait();
  const QkvShape& s = a.s;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int group = s.heads / s.kv_heads;
  const int hpb = min(group, kFaMaxHeads), n_hb = (group + hpb - 1) / hpb;
  const int tpb = kFaRows / hpb;  // tokens per CTA
  const int g = blockIdx.y / n_hb, hb = blockIdx.y - g * n_hb;
  const int h0 = g * group + hb * hpb, nh = min(hpb, group - hb * hpb);
  const int t0 = (gridDim.x - 1 - blockIdx.x) * tpb;  // the longest ranges first
  const int nt = min(tpb, a.rows - t0);
  const int pos0 = *a.pos;
  const int qp = s.dimp + 8, vpitch = s.vdimp + 8;
  __nv_bfloat16* qs = fsm;
  __nv_bfloat16* ks = qs + kFaRows * qp;
  __nv_bfloat16* vs = ks + 2 * kFaKeys * qp;
  const __nv_bfloat16* kc = a.k_cache + g * a.k_head;
  const __nv_bfloat16* vc = a.v_cache + g * a.v_head;
  const int lo = s.window > 0 ? max(0, pos0 + t0 - s.window + 1) : 0, hi = pos0 + t0 + nt;  // keys any row sees

  const int dch = s.dimp / 8;
  for (int i = tid; i < kFaRows * dch; i += kFaThreads) {
    const int r = i / dch, c = i - r * dch;
    const int tt = r / hpb, h = r - tt * hpb;
    const bool ok = tt < nt && h < nh;
    const long long row = ok ? static_cast<long long>(t0 + tt) * s.heads + h0 + h : 0;
    cp_async16(qs + r * qp + c * 8, a.q + row * s.dimp + c * 8, ok);
  }
  // rows k0 .. of the keys or values: ch1 pieces of eight from src1, the others from src2
  auto load_rows = [&](__nv_bfloat16* dst, int pitch, const __nv_bfloat16* src1, long long ld1, int ch1, const __nv_bfloat16* src2,
                       long long ld2, int ch, int k0) {
    const int slot0 = k0 % s.ring;
    for (int i = tid; i < kFaKeys * ch; i += kFaThreads) {
      const int r = i / ch, c = i - r * ch;
      const bool ok = k0 + r < hi;
      const long long slot = ok ? slot0 + r - (slot0 + r >= s.ring ? s.ring : 0) : 0;
      cp_async16(dst + r * pitch + c * 8, c < ch1 ? src1 + slot * ld1 + c * 8 : src2 + slot * ld2 + (c - ch1) * 8, ok);
    }
    cp_async_commit();
  };
  auto load_keys = [&](int buf, int k0) {
    load_rows(ks + buf * kFaKeys * qp, qp, kc, a.k_ld, a.dim1 / 8, a.k2, a.k2_ld, s.dimp / 8, k0);
  };
  auto load_values = [&](int k0) { load_rows(vs, vpitch, vc, a.v_ld, s.vdimp / 8, vc, a.v_ld, s.vdimp / 8, k0); };
  load_keys(0, lo);
  load_values(lo);

  float o[DV16 * 2][4];
#pragma unroll
  for (int i = 0; i < DV16 * 2; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) o[i][j] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  // this thread's two rows (lane / 4 and + 8 inside the warp's 16)
  int qpos[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = warp * 16 + (lane >> 2) + i * 8, tt = r / hpb;
    qpos[i] = tt < nt ? pos0 + t0 + tt : -1;  // a row without a token sees nothing
  }
  const int win = s.window > 0 ? s.window : 0x7fffffff;
  const int n_tiles = (hi - lo + kFaKeys - 1) / kFaKeys;
  for (int tile = 0; tile < n_tiles; ++tile) {
    const int k0 = lo + tile * kFaKeys, buf = tile & 1;
    const bool more = tile + 1 < n_tiles;
    cp_async_wait<1>();  // all but the newest group: this tile's keys (its values are the newest)
    __syncthreads();
    if (more) load_keys(buf ^ 1, k0 + kFaKeys);
    const __nv_bfloat16* kt = ks + buf * kFaKeys * qp;
    float sacc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) sacc[i][j] = 0.f;
    for (int kk = 0; kk < s.dimp / 16; ++kk) {
      uint32_t qa[4];
      ldmatrix_x4(qa, qs + (warp * 16 + (lane & 15)) * qp + kk * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int nb = 0; nb < 4; ++nb) {
        uint32_t kb[4];  // two tiles of eight keys: (k 0-7, k 8-15) each
        ldmatrix_x4(kb, kt + (nb * 16 + (lane & 7) + (lane >> 4) * 8) * qp + kk * 16 + ((lane >> 3) & 1) * 8);
        const uint32_t b0[2] = {kb[0], kb[1]}, b1[2] = {kb[2], kb[3]};
        mma_bf16_16816(sacc[nb * 2], qa, b0);
        mma_bf16_16816(sacc[nb * 2 + 1], qa, b1);
      }
    }
    float mx[2] = {-INFINITY, -INFINITY};
    // every key of an inner tile is visible to every row (rows without a token are never stored)
    const bool inner = k0 + kFaKeys - 1 <= pos0 + t0 && hi - 1 - k0 < win;
    if (inner) {
#pragma unroll
      for (int nt8 = 0; nt8 < 8; ++nt8)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          sacc[nt8][j] *= a.scale;
          mx[j >> 1] = fmaxf(mx[j >> 1], sacc[nt8][j]);
        }
    } else {
#pragma unroll
      for (int nt8 = 0; nt8 < 8; ++nt8)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int kpos = k0 + nt8 * 8 + (lane & 3) * 2 + (j & 1), i = j >> 1;
          const bool ok = kpos <= qpos[i] && qpos[i] - kpos < win;
          sacc[nt8][j] = ok ? sacc[nt8][j] * a.scale : -INFINITY;
          mx[i] = fmaxf(mx[i], sacc[nt8][j]);
        }
    }
    float corr[2], msafe[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
      const float mn = fmaxf(m[i], mx[i]);
      msafe[i] = mn == -INFINITY ? 0.f : mn;
      corr[i] = __expf(m[i] - msafe[i]);
      m[i] = mn;
      l[i] *= corr[i];
    }
#pragma unroll
    for (int i = 0; i < DV16 * 2; ++i) {
      o[i][0] *= corr[0];
      o[i][1] *= corr[0];
      o[i][2] *= corr[1];
      o[i][3] *= corr[1];
    }
    uint32_t pa[4][4];
#pragma unroll
    for (int nb = 0; nb < 4; ++nb) {
      float e[8];
#pragma unroll
      for (int q = 0; q < 2; ++q)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float v = __expf(sacc[nb * 2 + q][j] - msafe[j >> 1]);
          e[q * 4 + j] = v;
          l[j >> 1] += v;
        }
      pa[nb][0] = pack_bf16x2(e[0], e[1]);
      pa[nb][1] = pack_bf16x2(e[2], e[3]);
      pa[nb][2] = pack_bf16x2(e[4], e[5]);
      pa[nb][3] = pack_bf16x2(e[6], e[7]);
    }
    if (more) cp_async_wait<1>(); else cp_async_wait<0>();  // this tile's values
    __syncthreads();
#pragma unroll
    for (int vb = 0; vb < DV16; ++vb) {
      if (vb * 16 < s.vdimp) {
#pragma unroll
        for (int nb = 0; nb < 4; ++nb) {
          uint32_t bv[4];  // keys 0-7 / 8-15 of columns 0-7, then of columns 8-15
          ldmatrix_x4_trans(bv, vs + (nb * 16 + (lane & 15)) * vpitch + vb * 16 + (lane >> 4) * 8);
          const uint32_t b0[2] = {bv[0], bv[1]}, b1[2] = {bv[2], bv[3]};
          mma_bf16_16816(o[vb * 2], pa[nb], b0);
          mma_bf16_16816(o[vb * 2 + 1], pa[nb], b1);
        }
      }
    }
    __syncthreads();
    if (more) load_values(k0 + kFaKeys);
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
    const int r = warp * 16 + (lane >> 2) + i * 8, tt = r / hpb, h = r - tt * hpb;
    if (tt >= nt || h >= nh) continue;
    float inv = 1.f / l[i];
    if (a.sink != nullptr) {
      const float sk = a.sink[h0 + h], top = fmaxf(m[i], sk), e = expf(m[i] - top);
      inv = e / (l[i] * e + expf(sk - top));
    }
    if (a.gate.per_head) inv *= a.gate(t0 + tt, h0 + h, s.vdim, 0);
    const bool gated = a.gate.z != nullptr && !a.gate.per_head;
    __nv_bfloat16* dst = a.out + static_cast<long long>(t0 + tt) * a.ldo + (h0 + h) * s.vdim;
    const bool pairs = (s.vdim & 1) == 0;
#pragma unroll
    for (int vb = 0; vb < DV16 * 2; ++vb) {
      const int c = vb * 8 + (lane & 3) * 2;
      float o0 = o[vb][i * 2] * inv, o1 = o[vb][i * 2 + 1] * inv;
      if (gated) {
        if (c < s.vdim) o0 *= a.gate(t0 + tt, h0 + h, s.vdim, c);
        if (c + 1 < s.vdim) o1 *= a.gate(t0 + tt, h0 + h, s.vdim, c + 1);
      }
      if (pairs) {
        if (c < s.vdim) *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16x2(o0, o1);
      } else {
        if (c < s.vdim) dst[c] = f2bf(o0);
        if (c + 1 < s.vdim) dst[c + 1] = f2bf(o1);
      }
    }
  }
}

}  // namespace tb
