// Radix selection of the k largest values of one row by one CTA, on the order-preserving unsigned image of
// f32: exact, equal values by lower index first.  Shared by the indexer's selection and the token sampler.
#pragma once

#include "common.cuh"

namespace tb {

// ------------------------------------------------------------------ radix top-k
__device__ __forceinline__ uint32_t f32_order_key(float v) {
  uint32_t u = __float_as_uint(v);
  if (u == 0x80000000u) u = 0u;  // -0.0 compares equal to +0.0
  return (u & 0x80000000u) ? ~u : (u | 0x80000000u);
}
constexpr uint32_t kNegInfKey = 0x007fffffu;  // order key of -inf: never selected

constexpr int kTopkThreads = 1024;
constexpr int kTopkItems = 8;  // consecutive elements per thread in the ordered compaction

// One CTA per row.  Selects the k largest logits among [0, n) (entries equal to -inf are skipped),
// ties by lower index, and writes their indices in ascending order; unused slots get -1.
// The selection for one row by one CTA of kTopkThreads threads; `dst` may be shared or global memory.
template <int THREADS>
__device__ __forceinline__ void topk_radix_row(const float* row, int n, int k, int* dst) {
  constexpr int kTopkThreads = THREADS;  // shadows the launch constant: the strides below follow the caller's block
  __shared__ int hist[256];
  __shared__ uint32_t s_prefix;
  __shared__ int s_remaining;
  __shared__ int s_warp_gt[32], s_warp_eq[32];
  __shared__ int s_base_sel, s_base_eq;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;

  // count eligible entries
  int cnt = 0;
  for (int i = tid; i < n; i += kTopkThreads) cnt += f32_order_key(__ldcg(row + i)) > kNegInfKey;
  if (tid < 256) hist[tid] = 0;
  if (tid == 0) { s_prefix = 0; s_remaining = 0; }
  __syncthreads();
  {
    int wsum = cnt;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) wsum += __shfl_xor_sync(0xffffffffu, wsum, o);
    if (lane == 0) atomicAdd(&s_remaining, wsum);
  }
  __syncthreads();
  const int n_eligible = s_remaining;
  __syncthreads();

  uint32_t thr = kNegInfKey + 1;  // select everything eligible
  int need_eq = 0x7fffffff;       // how many entries equal to thr to take
  bool take_all = n_eligible <= k;
  if (!take_all) {
    if (tid == 0) s_remaining = k;
    __syncthreads();
    uint32_t prefix = 0, mask = 0;
    for (int shift = 24; shift >= 0; shift -= 8) {
      if (tid < 256) hist[tid] = 0;
      __syncthreads();
      for (int i = tid; i < n; i += kTopkThreads) {
        const uint32_t key = f32_order_key(__ldcg(row + i));
        if (key > kNegInfKey && (key & mask) == prefix) atomicAdd(&hist[(key >> shift) & 0xff], 1);
      }
      __syncthreads();
      if (warp == 0) {
        // find the digit where the count of larger-or-equal digits reaches the remaining quota:
        // lane l owns bins 8l .. 8l+7; suffix sums across lanes, then a short scan inside one lane
        const int rem = s_remaining;
        int b[8], ssum = 0;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          b[j] = hist[lane * 8 + j];
          ssum += b[j];
        }
        int suf = ssum;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const int v = __shfl_down_sync(0xffffffffu, suf, o);
          if (lane + o < 32) suf += v;
        }
        int suf_next = __shfl_down_sync(0xffffffffu, suf, 1);
        if (lane == 31) suf_next = 0;
        if (suf >= rem && suf_next < rem) {
          int r = rem - suf_next, d = 0;
          bool found = false;
#pragma unroll
          for (int j = 7; j >= 0; --j) {
            if (!found) {
              if (b[j] >= r || j == 0) {
                d = j;
                found = true;
              } else {
                r -= b[j];
              }
            }
          }
          s_remaining = r;
          s_prefix = prefix | (static_cast<uint32_t>(lane * 8 + d) << shift);
        }
      }
      __syncthreads();
      prefix = s_prefix;
      mask |= 0xffu << shift;
      __syncthreads();
    }
    thr = prefix;
    need_eq = s_remaining;
  }

  // ordered compaction: chunk of kTopkThreads * kTopkItems consecutive elements per pass
  if (tid == 0) { s_base_sel = 0; s_base_eq = 0; }
  __syncthreads();
  for (int base = 0; base < n; base += kTopkThreads * kTopkItems) {
    const int i0 = base + tid * kTopkItems;
    uint32_t gt_mask = 0, eq_mask = 0;
#pragma unroll
    for (int j = 0; j < kTopkItems; ++j) {
      const int i = i0 + j;
      if (i < n) {
        const uint32_t key = f32_order_key(__ldcg(row + i));
        if (key > kNegInfKey) {
          if (take_all || key > thr) gt_mask |= 1u << j;
          else if (key == thr) eq_mask |= 1u << j;
        }
      }
    }
    const int my_gt = __popc(gt_mask), my_eq = __popc(eq_mask);
    // exclusive scans of (gt, eq) over the CTA in thread order
    int sc_gt = my_gt, sc_eq = my_eq;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int a = __shfl_up_sync(0xffffffffu, sc_gt, o), b = __shfl_up_sync(0xffffffffu, sc_eq, o);
      if (lane >= o) { sc_gt += a; sc_eq += b; }
    }
    if (lane == 31) { s_warp_gt[warp] = sc_gt; s_warp_eq[warp] = sc_eq; }
    __syncthreads();
    int pre_gt = 0, pre_eq = 0, tot_gt = 0, tot_eq = 0;
    for (int w2 = 0; w2 < kTopkThreads / 32; ++w2) {
      const int a = s_warp_gt[w2], b = s_warp_eq[w2];
      if (w2 < warp) { pre_gt += a; pre_eq += b; }
      tot_gt += a; tot_eq += b;
    }
    const int base_sel = s_base_sel, base_eq = s_base_eq;
    // ties consumed before this thread (in index order) and how many of them were taken
    int eq_before = base_eq + pre_eq + sc_eq - my_eq;
    int gt_before = pre_gt + sc_gt - my_gt;
    // selected-so-far = base_sel (all earlier chunks) + gt in this chunk before me + ties taken in this chunk before me
    const int eq_taken_before_chunk = min(base_eq, need_eq);
    int eq_taken_before_me = min(eq_before, need_eq) - eq_taken_before_chunk;
    int w = base_sel + gt_before + eq_taken_before_me;
#pragma unroll
    for (int j = 0; j < kTopkItems; ++j) {
      if (gt_mask & (1u << j)) {
        if (w < k) dst[w] = i0 + j;
        ++w;
      } else if (eq_mask & (1u << j)) {
        if (eq_before < need_eq) {
          if (w < k) dst[w] = i0 + j;
          ++w;
        }
        ++eq_before;
      }
    }
    __syncthreads();
    if (tid == 0) {
      const int eq_taken_chunk = min(base_eq + tot_eq, need_eq) - eq_taken_before_chunk;
      s_base_sel = base_sel + tot_gt + eq_taken_chunk;
      s_base_eq = base_eq + tot_eq;
    }
    __syncthreads();
  }
  const int n_sel = s_base_sel;
  for (int i = n_sel + tid; i < k; i += kTopkThreads) dst[i] = -1;
}

}  // namespace tb
