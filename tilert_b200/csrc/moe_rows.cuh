// Routing of token rows to experts: the `top` largest router logits, softmax over the chosen ones only, the rank
// of every (token, expert) pair inside its expert's segment, and the gather of activation rows into expert order.
#pragma once

#include "act.cuh"

namespace tb {

constexpr int kRouteWarps = 8;
constexpr int kMaxExperts = 1024;
constexpr int kMaxTop = 32;

// One warp: the `top` largest of z[0..n) (equal values: lower index first) and the softmax over them.  z is
// overwritten.  ids / w are shared or global memory; every lane returns after they are written.
__device__ __forceinline__ void select_softmax_warp(float* z, int n, int top, int* ids, float* w) {
  const int lane = threadIdx.x & 31;
  for (int i = lane; i < n; i += 32) {
    const float v = z[i];
    z[i] = v >= -3.402823466e38f ? v : -3.402823466e38f;  // -inf and nan: the lowest value that is still selectable
  }
  __syncwarp();
  float zmax = 0.f, sum = 0.f;
  for (int j = 0; j < top; ++j) {
    float best = -INFINITY;
    int idx = 0x7fffffff;
    for (int i = lane; i < n; i += 32)
      if (z[i] > best) {
        best = z[i];
        idx = i;
      }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float b = __shfl_xor_sync(0xffffffffu, best, o);
      const int k = __shfl_xor_sync(0xffffffffu, idx, o);
      if (b > best || (b == best && k < idx)) {
        best = b;
        idx = k;
      }
    }
    if (j == 0) zmax = best;
    const float e = expf(best - zmax);
    sum += e;
    if (lane == 0) {
      ids[j] = idx;
      w[j] = e;
      z[idx] = -INFINITY;  // taken
    }
    __syncwarp();
  }
  for (int j = lane; j < top; j += 32) w[j] = w[j] / sum;
  __syncwarp();
}

struct RouteRowsParams {
  const float* logits;  // [rows, ldl], bias included
  long long ldl;
  int rows, n_experts, top;
  int* ids;             // [rows, top]
  float* w;             // [rows, top]
  int* rank;            // [rows, top] place inside the expert's segment
  int* counts;          // [n_experts], zero on entry
};

__global__ void __launch_bounds__(kRouteWarps * 32) route_rows_kernel(const RouteRowsParams p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float zs[];  // [kRouteWarps][n_experts]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * kRouteWarps + warp;
  if (t >= p.rows) return;
  float* z = zs + warp * p.n_experts;
  for (int i = lane; i < p.n_experts; i += 32) z[i] = p.logits[t * p.ldl + i];
  __syncwarp();
  int* ids = p.ids + t * p.top;
  select_softmax_warp(z, p.n_experts, p.top, ids, p.w + t * p.top);
  for (int j = lane; j < p.top; j += 32) p.rank[t * p.top + j] = atomicAdd(p.counts + ids[j], 1);
}

struct GatherRowsParams {
  const void* x;        // [rows, ldx]
  long long ldx;        // multiple of 8
  int dim8;             // 8-element pieces per row
  int top, n_experts;
  const int* ids;       // [rows, top]
  const int* rank;
  const int* counts;    // [n_experts]
  void* xs;             // [rows * top, ldx] in expert order
  int* slot_row;        // [rows, top]
};

template <typename T>
__global__ void __launch_bounds__(256) gather_rows_kernel(const GatherRowsParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  __shared__ int s_row[kMaxTop];
  for (int j = warp; j < p.top; j += blockDim.x >> 5) {
    const int e = p.ids[t * p.top + j];
    int base = 0;
    for (int i = lane; i < e; i += 32) base += p.counts[i];
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) base += __shfl_xor_sync(0xffffffffu, base, o);
    if (lane == 0) {
      const int row = base + p.rank[t * p.top + j];
      s_row[j] = row;
      p.slot_row[t * p.top + j] = row;
    }
  }
  __syncthreads();
  constexpr int kVec = 16 / sizeof(T);  // elements per 16 bytes
  const int n = p.dim8 * 8 / kVec;
  const uint4* src = reinterpret_cast<const uint4*>(reinterpret_cast<const T*>(p.x) + t * p.ldx);
  for (int c = threadIdx.x; c < n; c += blockDim.x) {
    const uint4 v = src[c];
    for (int j = 0; j < p.top; ++j)
      reinterpret_cast<uint4*>(reinterpret_cast<T*>(p.xs) + static_cast<long long>(s_row[j]) * p.ldx)[c] = v;
  }
}

}  // namespace tb
