// Single-token products: one activation vector (f32) against bf16 weights, bound by the weight stream from HBM.
//
//   dense     out[n] = W[n, :] . x (+ bias)
//   gated     hidden[n] = clamped_gate(W_gate[n, :] . x, W_up[n, :] . x)
//   gate/up   routing, then hidden = clamped_gate(W_gate x, W_up x) of the shared and the selected experts
//   down      out[d] = sum over slots of w_slot W_down[slot][d, :] . hidden[slot]
//
// One CTA of 16 warps per SM.  A CTA owns a contiguous range of weight rows.  A team of warps -- all 16, or fewer when
// K is short -- works on four rows at a time: its threads split K (piece c of eight elements belongs to thread c mod
// team size) and have the next two steps' rows already requested, so that 8-12 sixteen-byte loads per thread are in
// flight.  Four row sums are reduced across a warp together (transposing: six shuffles instead of twenty) and the
// per-warp sums of a team meet in shared memory at the end.
//
// The vector is staged once per CTA.  Staging can apply what lies between two sublayers -- x + norm(y) (+ a constant
// vector), written back by CTA 0, and a further norm on top -- so that the norms and the residual of a decode step need
// no launches of their own.  A norm is the RMS norm, or with `centered` the layer norm.  Weights that do not depend on
// the predecessor are requested before the wait for it.
#pragma once

#include "act.cuh"
#include "moe_rows.cuh"

namespace tb {

constexpr int kRvThreads = 512;
constexpr int kRvWarps = kRvThreads / 32;
constexpr int kRvRows = 4;
constexpr int kRvAhead = 2;        // steps requested beyond the current one
constexpr int kRvBatchRows = 512;  // weight rows between two reductions over the warps

struct RvStage {
  const float* x;      // [pad8(k)], zero beyond k, as are y and all constants
  const float* y;      // optional sublayer output: the vector is x + norm(y)
  const float* gain;   // with y
  const float* bias;   // optional, with y
  const float* add;    // optional constant added to the vector
  const float* gain2;  // optional norm of the result
  const float* bias2;  // optional, with gain2
  float* x_out;        // optional: CTA 0 stores the vector (before gain2); must not alias x or y
  float eps;
  int centered;        // both norms
  int k;
};

__host__ __device__ inline int rv_half_words(int kp) { return pad_to(kp / 2, 32) + 16; }  // keeps the halves 16 banks apart
__host__ __device__ inline size_t rv_vec_bytes(int kp) { return (rv_half_words(kp) + kp / 2) * sizeof(float); }
constexpr size_t kRvPartBytes = kRvBatchRows * kRvWarps * sizeof(float);

// The staged vector: elements 0-3 of every piece of eight in one half, 4-7 in the other, so that a warp's 16-byte
// reads are free of bank conflicts.
struct RvVec {
  float* lo;
  float* hi;
  __device__ __forceinline__ void put4(int g, const float4& v) const {  // g = element / 4
    reinterpret_cast<float4*>(g & 1 ? hi : lo)[g >> 1] = v;
  }
  __device__ __forceinline__ float4 get4(int g) const { return reinterpret_cast<const float4*>(g & 1 ? hi : lo)[g >> 1]; }
};

__device__ __forceinline__ float dot4(const float4& a) { return a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w; }
__device__ __forceinline__ float sum4(const float4& a) { return (a.x + a.y) + (a.z + a.w); }
// (v - mean) * rinv * gain + bias
__device__ __forceinline__ float4 norm4(const float4& v, float mean, float rinv, const float* gain, const float* bias, int g) {
  const float4 c = reinterpret_cast<const float4*>(gain)[g];
  const float4 b = bias != nullptr ? reinterpret_cast<const float4*>(bias)[g] : make_float4(0.f, 0.f, 0.f, 0.f);
  return make_float4((v.x - mean) * rinv * c.x + b.x, (v.y - mean) * rinv * c.y + b.y, (v.z - mean) * rinv * c.z + b.z,
                     (v.w - mean) * rinv * c.w + b.w);
}

// Statistics of the staged vector, every thread reading the groups it wrote itself; `first` is the thread's sum of
// values (centered) or of squares.
__device__ __forceinline__ void rv_stat(const RvVec& v, int k, float eps, int centered, float first, float* red, float& mean, float& rinv) {
  float ss = first;
  mean = 0.f;
  if (centered) {
    mean = cta_sum(first, red) / static_cast<float>(k);
    ss = 0.f;
    for (int g = threadIdx.x; g < pad_to(k, 8) / 4; g += kRvThreads) {
      const float4 a = v.get4(g);
      const float4 d = make_float4(a.x - mean, a.y - mean, a.z - mean, a.w - mean);
      if (4 * g + 4 <= k) {
        ss += dot4(d);
      } else {  // the padding is no value
        if (4 * g < k) ss += d.x * d.x;
        if (4 * g + 1 < k) ss += d.y * d.y;
        if (4 * g + 2 < k) ss += d.z * d.z;
      }
    }
  }
  rinv = 1.f / sqrtf(cta_sum(ss, red) / static_cast<float>(k) + eps);
}

// Constants of the staging, requested before the wait for the predecessor.
__device__ __forceinline__ void rv_prefetch(const RvStage& s) {
  const float* c[5] = {s.gain, s.bias, s.add, s.gain2, s.bias2};
  for (int i = threadIdx.x * 32; i < s.k; i += kRvThreads * 32)
#pragma unroll
    for (int j = 0; j < 5; ++j)
      if (c[j] != nullptr) asm volatile("prefetch.global.L1 [%0];" ::"l"(c[j] + i));
}

__device__ __forceinline__ void rv_stage(const RvStage& s, const RvVec& v, float* red) {
  constexpr int kReg = 4;  // groups of four per thread held in registers: k up to 8192 costs one round trip
  const int ng = pad_to(s.k, 8) / 4;
  const float4* x4 = reinterpret_cast<const float4*>(s.x);
  const float4* y4 = reinterpret_cast<const float4*>(s.y);
  float sum = 0.f, mean, rinv;
  auto finish = [&](int g, float4 o) {  // the vector's group g is known: into shared memory, and out
    if (s.add != nullptr) {
      const float4 c = reinterpret_cast<const float4*>(s.add)[g];
      o = make_float4(o.x + c.x, o.y + c.y, o.z + c.z, o.w + c.w);
    }
    v.put4(g, o);
    sum += s.centered ? sum4(o) : dot4(o);
    if (s.x_out != nullptr && blockIdx.x == 0) reinterpret_cast<float4*>(s.x_out)[g] = o;
  };
  if (s.y != nullptr) {
    float4 xr[kReg], yr[kReg];
#pragma unroll
    for (int i = 0; i < kReg; ++i) {
      const int g = threadIdx.x + i * kRvThreads;
      if (g < ng) {
        yr[i] = y4[g];
        xr[i] = x4[g];
      }
    }
    auto hold = [&](int g, const float4& a) {
      v.put4(g, a);
      sum += s.centered ? sum4(a) : dot4(a);
    };
#pragma unroll
    for (int i = 0; i < kReg; ++i)
      if (threadIdx.x + i * kRvThreads < ng) hold(threadIdx.x + i * kRvThreads, yr[i]);
    for (int g = threadIdx.x + kReg * kRvThreads; g < ng; g += kRvThreads) hold(g, y4[g]);
    rv_stat(v, s.k, s.eps, s.centered, sum, red, mean, rinv);
    sum = 0.f;
    auto emit = [&](int g, const float4& a) {
      const float4 n = norm4(v.get4(g), mean, rinv, s.gain, s.bias, g);
      finish(g, make_float4(a.x + n.x, a.y + n.y, a.z + n.z, a.w + n.w));
    };
#pragma unroll
    for (int i = 0; i < kReg; ++i)
      if (threadIdx.x + i * kRvThreads < ng) emit(threadIdx.x + i * kRvThreads, xr[i]);
    for (int g = threadIdx.x + kReg * kRvThreads; g < ng; g += kRvThreads) emit(g, x4[g]);
  } else {
#pragma unroll 4
    for (int g = threadIdx.x; g < ng; g += kRvThreads) finish(g, x4[g]);
  }
  if (s.gain2 != nullptr) {
    rv_stat(v, s.k, s.eps, s.centered, sum, red, mean, rinv);
    for (int g = threadIdx.x; g < ng; g += kRvThreads)  // every thread rescales what it wrote
      v.put4(g, norm4(v.get4(g), mean, rinv, s.gain2, s.bias2, g));
  }
  __syncthreads();
}

__device__ __forceinline__ uint4 ld_stream(const __nv_bfloat16* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}

// How the CTA's threads share rows of `chunks` pieces: teams of a power of two of warps, the smallest that
// covers a row in one go (or all of them).
struct RvTeam {
  int chunks, warps, threads, n_teams, team, tid, warp, nc;
  __device__ __forceinline__ explicit RvTeam(int chunks_) : chunks(chunks_) {
    warps = kRvWarps;
    while (warps > 1 && chunks <= warps * 16) warps >>= 1;
    threads = warps * 32;
    n_teams = kRvWarps / warps;
    team = threadIdx.x / threads;
    tid = threadIdx.x - team * threads;
    warp = tid >> 5;
    nc = (chunks + threads - 1) / threads;
  }
};

// Cursor over the (row group, piece) steps of a team.
struct RvCursor {
  int group, ci = 0;
  __device__ __forceinline__ explicit RvCursor(const RvTeam& t) : group(t.team) {}
  __device__ __forceinline__ void next(const RvTeam& t) {
    if (++ci == t.nc) {
      ci = 0;
      group += t.n_teams;
    }
  }
};

template <class Src>
__device__ __forceinline__ void rv_load(const Src& src, const RvTeam& t, const RvCursor& c, int rows, uint4 (&w)[kRvRows]) {
  const int piece = c.ci * t.threads + t.tid;
#pragma unroll
  for (int r = 0; r < kRvRows; ++r) {
    const int row = c.group * kRvRows + r;
    w[r] = (row < rows && piece < t.chunks) ? src.load(row, piece) : make_uint4(0u, 0u, 0u, 0u);
  }
}

// Sums of `rows` weight rows (Src::load(row, piece)) against the staged vector into part[row][warp of the team].
// `ahead` holds the first 1 + kRvAhead steps' weights when `loaded` is set.  vec(group) is the vector of a group of
// four rows.
template <class Src, class Vec>
__device__ __forceinline__ void rv_rows(const Src& src, const RvTeam& t, int rows, const Vec& vec, float* part,
                                        uint4 (&ahead)[kRvAhead + 1][kRvRows], bool loaded) {
  const int lane = threadIdx.x & 31;
  const int groups = (rows + kRvRows - 1) / kRvRows;
  const int steps = (groups - t.team + t.n_teams - 1) / t.n_teams * t.nc;  // of this team
  RvCursor cur(t), pre(t);
#pragma unroll
  for (int d = 0; d <= kRvAhead; ++d) {
    if (!loaded) rv_load(src, t, pre, rows, ahead[d]);
    pre.next(t);
  }
  float acc[kRvRows];
#pragma unroll
  for (int r = 0; r < kRvRows; ++r) acc[r] = 0.f;
#pragma unroll 3
  for (int s = 0; s < steps; ++s) {
    const int piece = cur.ci * t.threads + t.tid;
    if (piece < t.chunks) {
      const RvVec v = vec(cur.group);
      const float4 a = reinterpret_cast<const float4*>(v.lo)[piece], b = reinterpret_cast<const float4*>(v.hi)[piece];
#pragma unroll
      for (int r = 0; r < kRvRows; ++r) {
        float f[8];
        bf16x8_to_f32(ahead[0][r], f);
        acc[r] += f[0] * a.x + f[1] * a.y + f[2] * a.z + f[3] * a.w + f[4] * b.x + f[5] * b.y + f[6] * b.z + f[7] * b.w;
      }
    }
#pragma unroll
    for (int d = 0; d < kRvAhead; ++d)
#pragma unroll
      for (int r = 0; r < kRvRows; ++r) ahead[d][r] = ahead[d + 1][r];
    rv_load(src, t, pre, rows, ahead[kRvAhead]);
    pre.next(t);
    if (cur.ci == t.nc - 1) {
      // lanes 0 / 8 / 16 / 24 end up with the sums of rows 0 / 1 / 2 / 3
      const bool up16 = lane & 16, up8 = lane & 8;
      float a0 = (up16 ? acc[2] : acc[0]) + __shfl_xor_sync(0xffffffffu, up16 ? acc[0] : acc[2], 16);
      float a1 = (up16 ? acc[3] : acc[1]) + __shfl_xor_sync(0xffffffffu, up16 ? acc[1] : acc[3], 16);
      float b = (up8 ? a1 : a0) + __shfl_xor_sync(0xffffffffu, up8 ? a0 : a1, 8);
#pragma unroll
      for (int o = 4; o > 0; o >>= 1) b += __shfl_xor_sync(0xffffffffu, b, o);
      if ((lane & 7) == 0) part[(cur.group * kRvRows + (lane >> 3)) * kRvWarps + t.warp] = b;
#pragma unroll
      for (int r = 0; r < kRvRows; ++r) acc[r] = 0.f;
    }
    cur.next(t);
  }
}

struct RvOneVec {
  RvVec v;
  __device__ __forceinline__ RvVec operator()(int) const { return v; }
};

__device__ __forceinline__ float rv_total(const RvTeam& t, const float* part, int row) {
  float s = 0.f;
  if (t.warps >= 4) {
    const float4* q = reinterpret_cast<const float4*>(part + row * kRvWarps);
    for (int i = 0; i < t.warps / 4; ++i) s += (q[i].x + q[i].y) + (q[i].z + q[i].w);
  } else {
    for (int i = 0; i < t.warps; ++i) s += part[row * kRvWarps + i];
  }
  return s;
}

// ------------------------------------------------------------------ dense
struct RvDenseParams {
  RvStage in;
  const __nv_bfloat16* w;  // [n, ldw], ldw a multiple of 8 and >= pad8(k); columns beyond k are zero
  long long ldw;
  const float* bias;       // optional [n]
  int n;
  float* out;              // [n]
};

struct RvDenseSrc {
  const __nv_bfloat16* w;
  long long ldw;
  __device__ __forceinline__ uint4 load(int row, int piece) const { return ld_stream(w + row * ldw + piece * 8); }
};

__global__ void __launch_bounds__(kRvThreads, 1) rv_dense_kernel(const RvDenseParams p) {
  extern __shared__ __align__(16) float smem[];
  __shared__ float red[32];
  pdl_launch_dependents();
  const int kp = pad_to(p.in.k, 8);
  float* part = smem;
  const RvVec v{smem + kRvBatchRows * kRvWarps, smem + kRvBatchRows * kRvWarps + rv_half_words(kp)};
  const int r0 = static_cast<int>(static_cast<long long>(p.n) * blockIdx.x / gridDim.x);
  const int r1 = static_cast<int>(static_cast<long long>(p.n) * (blockIdx.x + 1) / gridDim.x);
  const RvTeam team(kp / 8);
  uint4 ahead[kRvAhead + 1][kRvRows];
  {
    const RvDenseSrc src{p.w + r0 * p.ldw, p.ldw};
    RvCursor c(team);
#pragma unroll
    for (int d = 0; d <= kRvAhead; ++d) {
      rv_load(src, team, c, min(r1 - r0, kRvBatchRows), ahead[d]);
      c.next(team);
    }
  }
  rv_prefetch(p.in);
  pdl_wait();
  rv_stage(p.in, v, red);
  for (int b = r0; b < r1; b += kRvBatchRows) {
    const int rows = min(r1 - b, kRvBatchRows);
    rv_rows(RvDenseSrc{p.w + b * p.ldw, p.ldw}, team, rows, RvOneVec{v}, part, ahead, b == r0);
    __syncthreads();
    for (int i = threadIdx.x; i < rows; i += kRvThreads) p.out[b + i] = rv_total(team, part, i) + (p.bias != nullptr ? p.bias[b + i] : 0.f);
    __syncthreads();
  }
}

// ------------------------------------------------------------------ gated halves of one dense feed-forward
struct RvGatedParams {
  RvStage in;
  const __nv_bfloat16* w;  // [2][n][ldw] (gate rows, then up rows)
  long long ldw;
  int n;
  float limit, alpha;
  float* out;              // [n]
};

struct RvGatedSrc {        // gate and up rows of a feature as neighbours
  const __nv_bfloat16* w;
  long long ldw, half;     // elements between the halves
  __device__ __forceinline__ uint4 load(int row, int piece) const { return ld_stream(w + (row & 1) * half + (row >> 1) * ldw + piece * 8); }
};

__global__ void __launch_bounds__(kRvThreads, 1) rv_gated_kernel(const RvGatedParams p) {
  extern __shared__ __align__(16) float smem[];
  __shared__ float red[32];
  pdl_launch_dependents();
  const int kp = pad_to(p.in.k, 8);
  float* part = smem;
  const RvVec v{smem + kRvBatchRows * kRvWarps, smem + kRvBatchRows * kRvWarps + rv_half_words(kp)};
  const int f0 = static_cast<int>(static_cast<long long>(p.n) * blockIdx.x / gridDim.x);
  const int f1 = static_cast<int>(static_cast<long long>(p.n) * (blockIdx.x + 1) / gridDim.x);
  const RvTeam team(kp / 8);
  const long long half = p.n * p.ldw;
  uint4 ahead[kRvAhead + 1][kRvRows];
  {
    const RvGatedSrc src{p.w + f0 * p.ldw, p.ldw, half};
    RvCursor c(team);
#pragma unroll
    for (int d = 0; d <= kRvAhead; ++d) {
      rv_load(src, team, c, min(2 * (f1 - f0), kRvBatchRows), ahead[d]);
      c.next(team);
    }
  }
  rv_prefetch(p.in);
  pdl_wait();
  rv_stage(p.in, v, red);
  for (int b = f0; b < f1; b += kRvBatchRows / 2) {
    const int feats = min(f1 - b, kRvBatchRows / 2);
    rv_rows(RvGatedSrc{p.w + b * p.ldw, p.ldw, half}, team, 2 * feats, RvOneVec{v}, part, ahead, b == f0);
    __syncthreads();
    for (int i = threadIdx.x; i < feats; i += kRvThreads)
      p.out[b + i] = clamped_gate(rv_total(team, part, 2 * i), rv_total(team, part, 2 * i + 1), p.limit, p.alpha);
    __syncthreads();
  }
}

// ------------------------------------------------------------------ experts: gate and up
struct RvGateUpParams {
  const float* x;              // [pad8(dim)] the sublayer's input
  int dim;
  const float* logits;         // [n_experts] router logits, bias included
  int n_experts, top;
  const __nv_bfloat16* w;      // [n_experts][2][ff][ldw] (gate rows, then up rows)
  const __nv_bfloat16* w_sh;   // [2][ff_sh][ldw] or null
  long long ldw;
  int ff, ff_sh;
  float limit, limit_sh, alpha;
  float* hidden;               // [pad8(ff_sh) + top * pad8(ff)], zero in the padding
  int* slot_ids;               // [top]
  float* slot_w;               // [top]
};

struct RvPtrSrc {
  const __nv_bfloat16* const* rows;
  __device__ __forceinline__ uint4 load(int row, int piece) const { return ld_stream(rows[row] + piece * 8); }
};

__global__ void __launch_bounds__(kRvThreads, 1) rv_gate_up_kernel(const RvGateUpParams p) {
  extern __shared__ __align__(16) float smem[];
  __shared__ float red[32];
  __shared__ int s_ids[kMaxTop];
  __shared__ float s_w[kMaxTop];
  __shared__ const __nv_bfloat16* s_row[kRvBatchRows];
  pdl_launch_dependents();
  const int kp = pad_to(p.dim, 8);
  float* part = smem;
  const RvVec v{smem + kRvBatchRows * kRvWarps, smem + kRvBatchRows * kRvWarps + rv_half_words(kp)};
  float* z = v.hi + kp / 2;
  pdl_wait();
  for (int i = threadIdx.x; i < p.n_experts; i += kRvThreads) z[i] = p.logits[i];
  RvStage in{};
  in.x = p.x;
  in.k = p.dim;
  rv_stage(in, v, red);
  if (threadIdx.x < 32) {
    select_softmax_warp(z, p.n_experts, p.top, s_ids, s_w);
    if (blockIdx.x == 0)
      for (int j = threadIdx.x; j < p.top; j += 32) {
        p.slot_ids[j] = s_ids[j];
        p.slot_w[j] = s_w[j];
      }
  }
  __syncthreads();
  const RvTeam team(kp / 8);
  const int n_feat = p.ff_sh + p.top * p.ff;
  const int f0 = static_cast<int>(static_cast<long long>(n_feat) * blockIdx.x / gridDim.x);
  const int f1 = static_cast<int>(static_cast<long long>(n_feat) * (blockIdx.x + 1) / gridDim.x);
  uint4 ahead[kRvAhead + 1][kRvRows];
  for (int b = f0; b < f1; b += kRvBatchRows / 2) {
    const int feats = min(f1 - b, kRvBatchRows / 2);
    for (int i = threadIdx.x; i < 2 * feats; i += kRvThreads) {
      const int f = b + (i >> 1), half = i & 1;
      if (f < p.ff_sh) {
        s_row[i] = p.w_sh + (static_cast<long long>(half) * p.ff_sh + f) * p.ldw;
      } else {
        const int j = (f - p.ff_sh) / p.ff, n = (f - p.ff_sh) - j * p.ff;
        s_row[i] = p.w + ((static_cast<long long>(s_ids[j]) * 2 + half) * p.ff + n) * p.ldw;
      }
    }
    __syncthreads();
    rv_rows(RvPtrSrc{s_row}, team, 2 * feats, RvOneVec{v}, part, ahead, false);
    __syncthreads();
    for (int i = threadIdx.x; i < feats; i += kRvThreads) {
      const int f = b + i;
      const bool shared = f < p.ff_sh;
      const int j = shared ? 0 : (f - p.ff_sh) / p.ff;
      const int dst = shared ? f : pad_to(p.ff_sh, 8) + j * pad_to(p.ff, 8) + (f - p.ff_sh) - j * p.ff;
      p.hidden[dst] = clamped_gate(rv_total(team, part, 2 * i), rv_total(team, part, 2 * i + 1), shared ? p.limit_sh : p.limit, p.alpha);
    }
    __syncthreads();
  }
}

// ------------------------------------------------------------------ experts: down
struct RvDownParams {
  const float* hidden;         // as written by the gate/up launch
  const int* slot_ids;
  const float* slot_w;
  int top;
  const __nv_bfloat16* w;      // [n_experts][dim][pad8(ff)], columns beyond ff zero
  const __nv_bfloat16* w_sh;   // [dim][pad8(ff_sh)] or null
  int ff, ff_sh, dim;
  float* out;                  // [dim]
};

struct RvPiece {
  const __nv_bfloat16* p;      // the piece in weight row 0
  long long ld;
};
struct RvPieceSrc {
  const RvPiece* pieces;
  int row0;
  __device__ __forceinline__ uint4 load(int row, int piece) const {
    return ld_stream(pieces[piece].p + (row0 + row) * pieces[piece].ld);
  }
};

__global__ void __launch_bounds__(kRvThreads, 1) rv_down_kernel(const RvDownParams p) {
  extern __shared__ __align__(16) float smem[];
  pdl_launch_dependents();
  const int ksh = pad_to(p.ff_sh, 8), ke = pad_to(p.ff, 8);
  const int kp = ksh + p.top * ke;
  float* part = smem;
  const RvVec v{smem + kRvBatchRows * kRvWarps, smem + kRvBatchRows * kRvWarps + rv_half_words(kp)};
  RvPiece* pieces = reinterpret_cast<RvPiece*>(v.hi + pad_to(kp / 2, 4));
  pdl_wait();
  for (int c = threadIdx.x; c < kp / 8; c += kRvThreads) {
    const bool shared = c * 8 < ksh;
    const int j = shared ? 0 : (c * 8 - ksh) / ke;
    const float w = shared ? 1.f : p.slot_w[j];
    pieces[c] = shared ? RvPiece{p.w_sh + c * 8, ksh}
                       : RvPiece{p.w + static_cast<long long>(p.slot_ids[j]) * p.dim * ke + (c * 8 - ksh - j * ke), ke};
    const float4* h = reinterpret_cast<const float4*>(p.hidden) + c * 2;
    const float4 a = h[0], b = h[1];
    v.put4(2 * c, make_float4(a.x * w, a.y * w, a.z * w, a.w * w));
    v.put4(2 * c + 1, make_float4(b.x * w, b.y * w, b.z * w, b.w * w));
  }
  __syncthreads();
  const int r0 = static_cast<int>(static_cast<long long>(p.dim) * blockIdx.x / gridDim.x);
  const int r1 = static_cast<int>(static_cast<long long>(p.dim) * (blockIdx.x + 1) / gridDim.x);
  const RvTeam team(kp / 8);
  uint4 ahead[kRvAhead + 1][kRvRows];
  for (int b = r0; b < r1; b += kRvBatchRows) {
    const int rows = min(r1 - b, kRvBatchRows);
    rv_rows(RvPieceSrc{pieces, b}, team, rows, RvOneVec{v}, part, ahead, false);
    __syncthreads();
    for (int i = threadIdx.x; i < rows; i += kRvThreads) p.out[b + i] = rv_total(team, part, i);
    __syncthreads();
  }
}

}  // namespace tb
