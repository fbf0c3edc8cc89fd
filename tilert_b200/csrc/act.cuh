// Activations are stored as bf16 or, for the exact mode, as f32; kernels that touch them are templates over the
// element type and use these helpers.  Vectors are padded with zeros to a multiple of eight elements (kActPad),
// so that rows can be read in 16-byte pieces whatever the model's sizes are.
#pragma once

#include "common.cuh"

namespace tb {

constexpr int kActPad = 8;
__host__ __device__ constexpr int pad_to(int n, int m) { return (n + m - 1) / m * m; }

__device__ __forceinline__ float act_ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ float act_ld(const float* p) { return *p; }
__device__ __forceinline__ void act_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void act_st(float* p, float v) { *p = v; }

__device__ __forceinline__ void bf16x8_to_f32(const uint4& u, float (&f)[8]) {
  f[0] = __uint_as_float(u.x << 16); f[1] = __uint_as_float(u.x & 0xffff0000u);
  f[2] = __uint_as_float(u.y << 16); f[3] = __uint_as_float(u.y & 0xffff0000u);
  f[4] = __uint_as_float(u.z << 16); f[5] = __uint_as_float(u.z & 0xffff0000u);
  f[6] = __uint_as_float(u.w << 16); f[7] = __uint_as_float(u.w & 0xffff0000u);
}
// eight consecutive elements (16-byte aligned)
__device__ __forceinline__ void act_ld8(const __nv_bfloat16* p, float (&f)[8]) {
  bf16x8_to_f32(*reinterpret_cast<const uint4*>(p), f);
}
__device__ __forceinline__ void act_ld8(const float* p, float (&f)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}

// Sum over the CTA (up to 32 warps); `red` holds 32 floats, every thread gets the sum.
__device__ __forceinline__ float cta_sum(float v, float* red) {
  const int lane = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  return warp_sum(lane < nw ? red[lane] : 0.f);
}

// The gated unit with clamped halves: g sigmoid(alpha g) (u + 1), g = min(gate, limit), u = up within +-limit.
__device__ __forceinline__ float clamped_gate(float gate, float up, float limit, float alpha) {
  const float g = fminf(gate, limit);
  const float u = fminf(fmaxf(up, -limit), limit);
  return g / (1.f + expf(-alpha * g)) * (u + 1.f);
}

// An output gate: one value per head, or one per element of every head.
struct HeadGate {
  const float* z;        // [rows, ld]; null: no gate
  long long ld;
  int per_head;
  __device__ __forceinline__ float operator()(int t, int h, int vdim, int v) const {
    return z == nullptr ? 1.f : 1.f / (1.f + expf(-z[t * ld + (per_head ? h : h * vdim + v)]));
  }
};

}  // namespace tb
