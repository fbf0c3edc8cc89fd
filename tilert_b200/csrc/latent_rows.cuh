// What surrounds attention over a latent cache, for a portion of tokens.  One row of the cache holds, for one position,
//
//   [ latent, RMS-normed (rank) | zeros to rankp | key part shared by all heads, rotated (rot) | zeros to row ]
//
// Keys and values are linear in the latent.  They can be expanded from it (expanded form), or the key expansion can be
// moved onto the query and the value expansion behind the sum (absorbed form): a query then is a row of the same layout,
// [W_uk^T q | zeros | rotated q | zeros], its score the dot product of two rows, and its result a sum of latents.
//
//   latent_tokens_kernel    the query latent normed, the cache row of every token
//   latent_queries_kernel   queries rotated and laid out for one of the forms
//   latent_merge_kernel     parts of an attention over key ranges (with a sink) -> sum of latents
//   gate_heads_kernel       head outputs times sigmoid(gate), heads side by side
#pragma once

#include "act.cuh"

namespace tb {

// A rotation of the first `dims` elements of a vector: pairs (2i, 2i + 1) when interleaved, else (i, i + dims / 2);
// table row p holds dims / 2 cosines, then dims / 2 sines, of position p.
struct Rotation {
  const float* table;
  int positions, dims, interleaved;

  // element e of the rotated vector, at(i) being element i of the vector
  template <class At>
  __device__ __forceinline__ float operator()(int pos, int e, At at) const {
    if (e >= dims) return at(e);
    const int half = dims / 2;
    const int i = interleaved ? e >> 1 : (e < half ? e : e - half);
    const bool second = interleaved ? (e & 1) != 0 : e >= half;
    const int partner = interleaved ? e ^ 1 : (second ? e - half : e + half);
    const float* row = table + static_cast<long long>(min(pos, positions - 1)) * dims;
    const float c = row[i], s = row[half + i];
    return second ? at(e) * c + at(partner) * s : at(e) * c - at(partner) * s;
  }
};

struct LatentRow {
  int rank, rankp, rot, row;  // rankp = rank padded to 16, row = rankp + rot padded to 32
};

struct LatentTokensParams {
  LatentRow r;
  Rotation rope;
  const float* z;        // [rows, ldz]: query latent (q_rank), at off_c the latent, at off_r the key part
  long long ldz;
  int q_rank, off_c, off_r;
  const float* q_gain;   // [q_rank]
  const float* c_gain;   // [rank]
  float eps;
  const int* pos;        // position of row 0
  int ring;
  void* cq;              // [rows, ldq] normed query latent
  long long ldq;
  void* cache;           // [ring, row]
};

template <typename T>
__global__ void __launch_bounds__(256) latent_tokens_kernel(const LatentTokensParams a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[32];
  const int t = blockIdx.x;
  const float* z = a.z + t * a.ldz;
  const float* c = z + a.off_c;
  const float* kr = z + a.off_r;
  float sq = 0.f, sc = 0.f;
  for (int i = threadIdx.x; i < a.q_rank; i += 256) sq += z[i] * z[i];
  for (int i = threadIdx.x; i < a.r.rank; i += 256) sc += c[i] * c[i];
  const float rq = 1.f / sqrtf(cta_sum(sq, red) / static_cast<float>(a.q_rank) + a.eps);
  const float rc = 1.f / sqrtf(cta_sum(sc, red) / static_cast<float>(a.r.rank) + a.eps);
  T* cq = reinterpret_cast<T*>(a.cq) + t * a.ldq;
  for (int i = threadIdx.x; i < a.q_rank; i += 256) act_st(cq + i, z[i] * rq * a.q_gain[i]);
  const int pos = *a.pos + t;
  T* dst = reinterpret_cast<T*>(a.cache) + static_cast<long long>(pos % a.ring) * a.r.row;
  for (int i = threadIdx.x; i < a.r.rank; i += 256) act_st(dst + i, c[i] * rc * a.c_gain[i]);
  for (int e = threadIdx.x; e < a.r.rot; e += 256) act_st(dst + a.r.rankp + e, a.rope(pos, e, [&](int i) { return kr[i]; }));
}

struct LatentQueriesParams {
  Rotation rope;
  const float* q;        // [rows, ldq]: per head `ldh` elements, dim unrotated and, at dimp8, rot to be rotated
  long long ldq;
  int heads, dim, dimp8, rot, ldh;
  const int* pos;
  int rows;
  // expanded form: out [rows, heads, wide], the rotated part at off_rot
  // absorbed form: the unrotated part to out [heads, rows, dimp8], the rotated one to lat [heads, rows, row] at off_rot
  void* out;
  int wide;
  int off_rot;
  float* lat;            // null: expanded form
  int row;
};

template <typename T>
__global__ void __launch_bounds__(256) latent_queries_kernel(const LatentQueriesParams a) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, pos = *a.pos + t, per = a.dim + a.rot;
  const float* q = a.q + t * a.ldq;
  T* out = reinterpret_cast<T*>(a.out);
  for (int i = threadIdx.x; i < a.heads * per; i += 256) {
    const int h = i / per, d = i - h * per;
    const float* src = q + h * a.ldh;
    const long long hr = a.lat != nullptr ? static_cast<long long>(h) * a.rows + t : static_cast<long long>(t) * a.heads + h;
    if (d < a.dim) {
      act_st(out + hr * (a.lat != nullptr ? a.dimp8 : a.wide) + d, src[d]);
    } else {
      const float v = a.rope(pos, d - a.dim, [&](int e) { return src[a.dimp8 + e]; });
      if (a.lat != nullptr)
        a.lat[hr * a.row + a.off_rot + d - a.dim] = v;
      else
        act_st(out + hr * a.wide + a.off_rot + d - a.dim, v);
    }
  }
}

// Weights of the parts of one query row: exp(max of the part - overall max) / overall sum; the sink is one more term of
// the sum.  By one warp; ml holds (max, sum) of every part, an empty part has max -inf.
__device__ __forceinline__ void part_weights(const float* ml, int n_splits, const float* sink, float* wgt) {
  const int lane = threadIdx.x & 31;
  float m = sink != nullptr ? *sink : -INFINITY, l = 0.f;
  for (int k = lane; k < n_splits; k += 32) m = fmaxf(m, ml[2 * k]);
  m = warp_max(m);
  for (int k = lane; k < n_splits; k += 32) l += expf(ml[2 * k] - m) * ml[2 * k + 1];
  l = warp_sum(l) + (sink != nullptr ? expf(*sink - m) : 0.f);
  for (int k = lane; k < n_splits; k += 32) wgt[k] = expf(ml[2 * k] - m) / l;
}
// Element groups of four of the merged row; a part of weight zero may hold anything.
__device__ __forceinline__ float4 merged4(const float* part, const float* wgt, int n_splits, int rankp, int g) {
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
  for (int k = 0; k < n_splits; ++k) {
    const float w = wgt[k];
    const float4 v = reinterpret_cast<const float4*>(part + static_cast<long long>(k) * rankp)[g];
    if (w != 0.f) o = make_float4(o.x + w * v.x, o.y + w * v.y, o.z + w * v.z, o.w + w * v.w);
  }
  return o;
}

struct LatentMergeParams {
  const float* part;     // [n_rows, n_splits, rankp], then [n_rows, n_splits, 2]
  int n_rows, tokens, n_splits, rank, rankp;
  const float* sink;     // optional [heads]
  void* out;             // [n_rows, ldo]
  long long ldo;
};

template <typename T>
__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentMergeParams a) {
  extern __shared__ __align__(16) float wgt[];  // [n_splits]
  pdl_launch_dependents();
  pdl_wait();
  const long long r = blockIdx.x;
  const float* ml = a.part + static_cast<long long>(a.n_rows) * a.n_splits * a.rankp + r * a.n_splits * 2;
  if (threadIdx.x < 32) part_weights(ml, a.n_splits, a.sink != nullptr ? a.sink + r / a.tokens : nullptr, wgt);
  __syncthreads();
  T* out = reinterpret_cast<T*>(a.out) + r * a.ldo;
  for (int g = threadIdx.x; g < a.rankp / 4; g += 128) {
    const float4 o = merged4(a.part + r * a.n_splits * a.rankp, wgt, a.n_splits, a.rankp, g);
    const float f[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (4 * g + j < a.rank) act_st(out + 4 * g + j, f[j]);
  }
}

struct GateHeadsParams {
  const float* o;        // [heads, rows, ldv]
  int ldv, heads, vdim, rows;
  HeadGate gate;
  void* out;             // [rows, ldo]
  long long ldo;
};

template <typename T>
__global__ void __launch_bounds__(256) gate_heads_kernel(const GateHeadsParams a) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  T* out = reinterpret_cast<T*>(a.out) + t * a.ldo;
  for (int i = threadIdx.x; i < a.heads * a.vdim; i += 256) {
    const int h = i / a.vdim, v = i - h * a.vdim;
    act_st(out + i, a.o[(static_cast<long long>(h) * a.rows + t) * a.ldv + v] * a.gate(t, h, a.vdim, v));
  }
}

}  // namespace tb
