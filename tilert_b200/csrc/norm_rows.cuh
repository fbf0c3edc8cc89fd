// Row kernels around the norms of a residual stream kept in f32: embedding + norm, sublayer output -> norm ->
// residual (-> norm of the next sublayer's input), and the norm in front of the vocabulary head.  One CTA per token; the
// gain vectors are f32 and already hold the factor the norm multiplies with (a weight that is an offset from one arrives
// as 1 + w).  A norm is the RMS norm, or with `centered` the layer norm (mean taken off first); biases are optional.
#pragma once

#include "act.cuh"

namespace tb {

constexpr int kNormThreads = 256;

struct RowStat {
  float mean, rinv;
};

// Statistics of n values that get(i) returns, the calling thread owning i = threadIdx.x, + blockDim.x, ...  The squared
// deviations are summed in a pass of their own (no cancellation).
template <class Get>
__device__ __forceinline__ RowStat row_stat(int n, float eps, int centered, float* red, Get get) {
  float mean = 0.f;
  if (centered) {
    float s = 0.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) s += get(i);
    mean = cta_sum(s, red) / static_cast<float>(n);
  }
  float ss = 0.f;
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const float d = get(i) - mean;
    ss += d * d;
  }
  return {mean, 1.f / sqrtf(cta_sum(ss, red) / static_cast<float>(n) + eps)};
}
__device__ __forceinline__ float row_norm(float v, const RowStat& st, const float* gain, const float* bias, int i) {
  return (v - st.mean) * st.rinv * gain[i] + (bias != nullptr ? bias[i] : 0.f);
}

struct EmbedNormParams {
  const long long* tokens;      // [rows]
  const __nv_bfloat16* table;   // [vocab, ld_table]
  long long ld_table;
  int vocab;
  const float* gain;            // null: the embedding as it is
  float eps;
  int dim;
  float* x;                     // [rows, ldx] f32 residual
  long long ldx;
  void* xh;                     // optional [rows, ldh] activations
  long long ldh;
  int* status;
};

template <typename T>
__global__ void __launch_bounds__(kNormThreads) embed_norm_kernel(const EmbedNormParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[32];
  const int t = blockIdx.x;
  const long long tok = p.tokens[t];
  if (tok < 0 || tok >= p.vocab) {  // uniform over the CTA
    if (threadIdx.x == 0) set_status(p.status, ST_BAD_ARGUMENT);
    return;
  }
  const __nv_bfloat16* row = p.table + tok * p.ld_table;
  RowStat st{0.f, 1.f};
  if (p.gain != nullptr) st = row_stat(p.dim, p.eps, 0, red, [&](int i) { return bf2f(row[i]); });
  for (int i = threadIdx.x; i < p.dim; i += kNormThreads) {
    const float v = p.gain != nullptr ? row_norm(bf2f(row[i]), st, p.gain, nullptr, i) : bf2f(row[i]);
    p.x[t * p.ldx + i] = v;
    if (p.xh != nullptr) act_st(reinterpret_cast<T*>(p.xh) + t * p.ldh + i, v);
  }
}

// x[t] += norm(y[t]) (+ add), where the sublayer output y is either one row, or a weighted sum of rows of expert
// outputs (row slot_row[t, j], weight slot_w[t, j]) plus an optional further row (a shared expert), or absent.  xh is
// x, or its norm with gain2.
struct ResidualNormParams {
  const float* y;               // [rows, ldy] f32, or null with slots
  long long ldy;
  const void* ye;               // expert outputs [*, lde], element type T
  long long lde;
  const int* slot_row;          // [rows, top]
  const float* slot_w;          // [rows, top]
  int top;
  const void* ysh;              // optional [rows, ldsh], element type T
  long long ldsh;
  const float* gain;            // null: no sublayer output
  const float* bias;            // optional
  const float* add;             // optional [dim], the same for every row
  const float* gain2;           // optional norm of the new x, for xh alone
  const float* bias2;           // optional
  int centered;                 // both norms
  float eps;
  int dim;
  float* x;                     // [rows, ldx] f32, updated
  long long ldx;
  void* xh;                     // optional [rows, ldh] x (or its norm) as activations
  long long ldh;
};

template <typename T>
__global__ void __launch_bounds__(kNormThreads) residual_norm_kernel(const ResidualNormParams p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float vals[];  // [dim]
  __shared__ float red[32];
  const int t = blockIdx.x;
  if (p.y != nullptr) {
    const float* y = p.y + t * p.ldy;
    for (int i = threadIdx.x; i < p.dim; i += kNormThreads) vals[i] = y[i];
  } else if (p.ye != nullptr) {
    const int n8 = pad_to(p.dim, 8) / 8;
    for (int c = threadIdx.x; c < n8; c += kNormThreads) {
      float acc[8];
#pragma unroll
      for (int q = 0; q < 8; ++q) acc[q] = 0.f;
      for (int j = 0; j < p.top; ++j) {
        const float w = p.slot_w[t * p.top + j];
        float f[8];
        act_ld8(reinterpret_cast<const T*>(p.ye) + static_cast<long long>(p.slot_row[t * p.top + j]) * p.lde + c * 8, f);
#pragma unroll
        for (int q = 0; q < 8; ++q) acc[q] += w * f[q];
      }
      if (p.ysh != nullptr) {
        float f[8];
        act_ld8(reinterpret_cast<const T*>(p.ysh) + t * p.ldsh + c * 8, f);
#pragma unroll
        for (int q = 0; q < 8; ++q) acc[q] += f[q];
      }
#pragma unroll
      for (int q = 0; q < 8; ++q)
        if (c * 8 + q < p.dim) vals[c * 8 + q] = acc[q];
    }
    __syncthreads();  // the pieces were eight wide
  }
  RowStat st{0.f, 0.f};
  if (p.gain != nullptr) st = row_stat(p.dim, p.eps, p.centered, red, [&](int i) { return vals[i]; });
  float* x = p.x + t * p.ldx;
  T* xh = p.xh != nullptr ? reinterpret_cast<T*>(p.xh) + t * p.ldh : nullptr;
  for (int i = threadIdx.x; i < p.dim; i += kNormThreads) {
    float v = x[i];
    if (p.gain != nullptr) v += row_norm(vals[i], st, p.gain, p.bias, i);
    if (p.add != nullptr) v += p.add[i];
    x[i] = v;
    if (p.gain2 != nullptr)
      vals[i] = v;
    else if (xh != nullptr)
      act_st(xh + i, v);
  }
  if (p.gain2 == nullptr) return;
  const RowStat s2 = row_stat(p.dim, p.eps, p.centered, red, [&](int i) { return vals[i]; });
  for (int i = threadIdx.x; i < p.dim; i += kNormThreads) act_st(xh + i, row_norm(vals[i], s2, p.gain2, p.bias2, i));
}

// out[r] = norm(x[rows[r]])
struct GatherNormParams {
  const float* x;
  long long ldx;
  const int* rows;              // [n]
  const float* gain;
  const float* bias;            // optional
  int centered;
  float eps;
  int dim;
  void* out;                    // [n, ldo]
  long long ldo;
};

template <typename T>
__global__ void __launch_bounds__(kNormThreads) gather_norm_kernel(const GatherNormParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[32];
  const float* x = p.x + static_cast<long long>(p.rows[blockIdx.x]) * p.ldx;
  const RowStat st = row_stat(p.dim, p.eps, p.centered, red, [&](int i) { return x[i]; });
  T* o = reinterpret_cast<T*>(p.out) + blockIdx.x * p.ldo;
  for (int i = threadIdx.x; i < p.dim; i += kNormThreads) act_st(o + i, row_norm(x[i], st, p.gain, p.bias, i));
}

}  // namespace tb
