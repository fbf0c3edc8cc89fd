// Row kernels around the norms of a residual stream kept in f32: embedding + norm, sublayer output -> norm ->
// residual, and the norm in front of the vocabulary head.  One CTA per token; the gain vectors are f32 and already
// hold the factor the norm multiplies with (a weight that is an offset from one arrives as 1 + w).
#pragma once

#include "act.cuh"

namespace tb {

constexpr int kNormThreads = 256;

struct EmbedNormParams {
  const long long* tokens;      // [rows]
  const __nv_bfloat16* table;   // [vocab, ld_table]
  long long ld_table;
  int vocab;
  const float* gain;
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
  float ss = 0.f;
  for (int i = threadIdx.x; i < p.dim; i += kNormThreads) {
    const float v = bf2f(row[i]);
    ss += v * v;
  }
  const float rinv = 1.f / sqrtf(cta_sum(ss, red) / static_cast<float>(p.dim) + p.eps);
  for (int i = threadIdx.x; i < p.dim; i += kNormThreads) {
    const float v = bf2f(row[i]) * rinv * p.gain[i];
    p.x[t * p.ldx + i] = v;
    if (p.xh != nullptr) act_st(reinterpret_cast<T*>(p.xh) + t * p.ldh + i, v);
  }
}

// x[t] += rms(y[t]) * gain, where the sublayer output y is either one row, or a weighted sum of rows of expert
// outputs (row slot_row[t, j], weight slot_w[t, j]) plus an optional further row (a shared expert).
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
  const float* gain;
  float eps;
  int dim;
  float* x;                     // [rows, ldx] f32, updated
  long long ldx;
  void* xh;                     // [rows, ldh] copy as activations
  long long ldh;
};

template <typename T>
__global__ void __launch_bounds__(kNormThreads) residual_norm_kernel(const ResidualNormParams p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float vals[];  // [dim]
  __shared__ float red[32];
  const int t = blockIdx.x;
  float ss = 0.f;
  if (p.y != nullptr) {
    const float* y = p.y + t * p.ldy;
    for (int i = threadIdx.x; i < p.dim; i += kNormThreads) {
      const float v = y[i];
      vals[i] = v;
      ss += v * v;
    }
  } else {
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
        if (c * 8 + q < p.dim) {
          vals[c * 8 + q] = acc[q];
          ss += acc[q] * acc[q];
        }
    }
  }
  const float rinv = 1.f / sqrtf(cta_sum(ss, red) / static_cast<float>(p.dim) + p.eps);  // (synchronises vals too)
  float* x = p.x + t * p.ldx;
  T* xh = reinterpret_cast<T*>(p.xh) + t * p.ldh;
  for (int i = threadIdx.x; i < p.dim; i += kNormThreads) {
    const float v = x[i] + vals[i] * rinv * p.gain[i];
    x[i] = v;
    act_st(xh + i, v);
  }
}

// out[r] = rms(x[rows[r]]) * gain
struct GatherNormParams {
  const float* x;
  long long ldx;
  const int* rows;              // [n]
  const float* gain;
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
  float ss = 0.f;
  for (int i = threadIdx.x; i < p.dim; i += kNormThreads) ss += x[i] * x[i];
  const float rinv = 1.f / sqrtf(cta_sum(ss, red) / static_cast<float>(p.dim) + p.eps);
  T* o = reinterpret_cast<T*>(p.out) + blockIdx.x * p.ldo;
  for (int i = threadIdx.x; i < p.dim; i += kNormThreads) act_st(o + i, x[i] * rinv * p.gain[i]);
}

}  // namespace tb
