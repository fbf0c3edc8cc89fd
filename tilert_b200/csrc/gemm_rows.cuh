// Products of many token rows with bf16 weights (prefill):  out[t, n] = W[n, :] . x[t, :].
//
//   gemm_tc_kernel<BN, GATED>   bf16 rows on the tensor cores
//   gemm_f32_kernel<GATED>      f32 rows, f32 arithmetic (the exact mode)
//
// GATED: the weight holds gate rows, then up rows, and the result is their clamped gated unit.
// Grouped launches have one weight per group (expert) and the token rows sorted by group; the number of rows per
// group is device data, so the tiles are enumerated on the device and the grid is the SM count.
//
// Tensor-core kernel: persistent, warp-specialised, one CTA per SM.  The 128 weight rows of a tile are M (so a TMEM
// lane is an output feature and a store covers consecutive features), BN token rows are N; K goes by 64.  One thread
// issues the TMA loads (128-byte swizzle) into a ring of stages, one thread issues the tcgen05.mma, eight warps read
// the accumulators back; two accumulators alternate so that the epilogue of a tile overlaps the products of the next.
#pragma once

#include <cuda.h>

#include "act.cuh"
#include "tcgen05.cuh"

namespace tb {

constexpr int kMaxGroups = 1024;

struct GemmRowsParams {
  int n;                 // output features
  int k;
  int rows;              // token rows; grouped with counts: an upper bound is not needed, the counts say how many
  int n_groups;          // 0: one weight for all rows
  const int* counts;     // [n_groups] device; null: `rows` rows in every group
  float limit, alpha;    // GATED
  const float* bias;     // optional [n] (one weight only)
  void* out;
  long long ldo;
  int out_bf16;
  int* status;
  // the exact mode reads its operands directly
  const __nv_bfloat16* w;
  long long ldw;
  const float* x;
  long long ldx;
};

// Enumeration of (group, feature tile, token tile); token tiles vary fastest, so that CTAs running together share a
// weight tile.  `rows0` / `tiles0` are exclusive prefix sums over the groups in shared memory.
struct TileWalk {
  const int* rows0;
  const int* tiles0;
  int n_groups, ft, bn;
  int group = 0;

  struct Tile {
    int group, feature0, row0, row1;
  };
  __device__ __forceinline__ Tile at(int i) {  // i must not decrease between calls
    while (i >= tiles0[group + 1]) ++group;
    const int local = i - tiles0[group], r0 = rows0[group], r1 = rows0[group + 1];
    const int tt = (r1 - r0 + bn - 1) / bn;
    const int f = local / tt, t = local - f * tt;
    return {group, f * 128, r0 + t * bn, min(r0 + (t + 1) * bn, r1)};
  }
};

// Fills the prefix sums (all threads of the CTA; s_rows / s_tiles hold max(n_groups, 1) + 1 entries).
__device__ __forceinline__ void tile_prefix(const GemmRowsParams& p, int bn, int ft, int* s_rows, int* s_tiles) {
  if (p.n_groups == 0) {
    if (threadIdx.x == 0) {
      s_rows[0] = s_tiles[0] = 0;
      s_rows[1] = p.rows;
      s_tiles[1] = (p.rows + bn - 1) / bn * ft;
    }
  } else if (threadIdx.x < 32) {
    int r0 = 0, t0 = 0;
    for (int b = 0; b < p.n_groups; b += 32) {
      const int e = b + static_cast<int>(threadIdx.x);
      const int c = e >= p.n_groups ? 0 : (p.counts != nullptr ? p.counts[e] : p.rows);
      int r = c, t = (c + bn - 1) / bn * ft;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int ra = __shfl_up_sync(0xffffffffu, r, o), ta = __shfl_up_sync(0xffffffffu, t, o);
        if (static_cast<int>(threadIdx.x) >= o) {
          r += ra;
          t += ta;
        }
      }
      if (e < p.n_groups) {
        s_rows[e + 1] = r0 + r;
        s_tiles[e + 1] = t0 + t;
      }
      r0 += __shfl_sync(0xffffffffu, r, 31);
      t0 += __shfl_sync(0xffffffffu, t, 31);
    }
    if (threadIdx.x == 0) s_rows[0] = s_tiles[0] = 0;
  }
  __syncthreads();
}

// ------------------------------------------------------------------ tensor cores
constexpr int kTcEpiWarps = 8;  // two per quarter of the TMEM lanes, each with half of the columns
constexpr int kTcThreads = 64 + 32 * kTcEpiWarps;  // and a producer warp, an MMA warp
constexpr int kTcK = 64;

template <int BN, bool GATED>
struct TcShape {
  static constexpr int kWBytes = 128 * kTcK * 2;
  static constexpr int kXBytes = BN * kTcK * 2;
  static constexpr int kStageBytes = (GATED ? 2 : 1) * kWBytes + kXBytes;
  static constexpr int kStages = 196608 / kStageBytes < 8 ? 196608 / kStageBytes : 8;
  static constexpr int kAccCols = GATED ? 2 * BN : BN;
  static constexpr int kTmemCols = 2 * kAccCols;
  static_assert(kTmemCols >= 32 && kTmemCols <= 512 && (kTmemCols & (kTmemCols - 1)) == 0, "TMEM allocation size");
  static constexpr size_t kSmemBytes = static_cast<size_t>(kStages) * kStageBytes + 1024;  // + alignment of the ring
};

// K-major operand in 128-byte swizzled rows (the layout a 64-element wide TMA box leaves): eight-row groups are
// 1024 bytes apart.
__device__ __forceinline__ uint64_t umma_desc_sw128(uint32_t smem_addr) {
  return static_cast<uint64_t>((smem_addr >> 4) & 0x3fffu) | (1ull << 16) | (static_cast<uint64_t>(1024 >> 4) << 32) | (1ull << 46) |
         (2ull << 61);
}
// D = f32, A = B = bf16, both K-major
__host__ __device__ constexpr uint32_t umma_idesc_bf16(int m, int n) {
  return (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(n >> 3) << 17) | (static_cast<uint32_t>(m >> 4) << 24);
}
__device__ __forceinline__ void umma_bf16(uint32_t tmem_d, uint64_t adesc, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}" ::"r"(tmem_d), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}
__device__ __forceinline__ void tma_load_2d(void* dst, const CUtensorMap* map, int x, int y, uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];" ::"r"(smem_u32(dst)),
      "l"(map), "r"(smem_u32(bar)), "r"(x), "r"(y)
      : "memory");
}
__device__ __forceinline__ void tmem_ld16(uint32_t taddr, uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]),
        "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(taddr));
}
// Completion of the loads issued so far; the registers are operands so that no use moves above it.
__device__ __forceinline__ void tmem_ld16_wait(uint32_t (&r)[16]) {
  asm volatile("tcgen05.wait::ld.sync.aligned;"
               : "+r"(r[0]), "+r"(r[1]), "+r"(r[2]), "+r"(r[3]), "+r"(r[4]), "+r"(r[5]), "+r"(r[6]), "+r"(r[7]), "+r"(r[8]), "+r"(r[9]),
                 "+r"(r[10]), "+r"(r[11]), "+r"(r[12]), "+r"(r[13]), "+r"(r[14]), "+r"(r[15])
               :
               : "memory");
}

// Lane l holds v[t], t = 0 .. 7, of feature l; returns the eight features of the lane's group of eight lanes for token
// l & 7.  Three exchanges, each between lanes one bit apart, each sending what the partner keeps.
__device__ __forceinline__ uint4 turn_eight(const float* v, int lane) {
  const bool b0 = lane & 1, b1 = lane & 2, b2 = lane & 4;
  uint32_t w[4];         // two features; w[k] of token 2 k + b0
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const float got = __shfl_xor_sync(0xffffffffu, b0 ? v[2 * k] : v[2 * k + 1], 1);
    w[k] = b0 ? pack_bf16x2(got, v[2 * k + 1]) : pack_bf16x2(v[2 * k], got);
  }
  uint32_t lo[2], hi[2];  // four features; of token 4 m + 2 b1 + b0
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    const uint32_t got = __shfl_xor_sync(0xffffffffu, b1 ? w[2 * m] : w[2 * m + 1], 2);
    lo[m] = b1 ? got : w[2 * m];
    hi[m] = b1 ? w[2 * m + 1] : got;
  }
  const uint32_t g0 = __shfl_xor_sync(0xffffffffu, b2 ? lo[0] : lo[1], 4), g1 = __shfl_xor_sync(0xffffffffu, b2 ? hi[0] : hi[1], 4);
  return b2 ? make_uint4(g0, g1, lo[1], hi[1]) : make_uint4(lo[0], hi[0], g0, g1);
}

template <int BN, bool GATED>
__global__ void __launch_bounds__(kTcThreads, 1)
    gemm_tc_kernel(const __grid_constant__ CUtensorMap wmap, const __grid_constant__ CUtensorMap xmap, const GemmRowsParams p) {
  using S = TcShape<BN, GATED>;
  extern __shared__ uint8_t smem_raw[];
  __shared__ __align__(8) uint64_t full[S::kStages], empty[S::kStages], acc_full[2], acc_empty[2], drain;
  __shared__ uint32_t s_tmem;
  __shared__ int s_abort;
  __shared__ int s_rows[kMaxGroups + 1], s_tiles[kMaxGroups + 1];
  uint8_t* ring = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  pdl_launch_dependents();
  if (threadIdx.x == 0) {
    for (int i = 0; i < S::kStages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&acc_full[i], 1);
      mbar_init(&acc_empty[i], kTcEpiWarps);
    }
    mbar_init(&drain, 1);
    s_abort = 0;
    mbar_fence_init();
  }
  if (warp == 2) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem)), "r"(S::kTmemCols)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(&s_tmem);
  pdl_wait();
  const int ft = (p.n + 127) / 128;
  tile_prefix(p, BN, ft, s_rows, s_tiles);
  const int groups = p.n_groups > 0 ? p.n_groups : 1;
  const int n_tiles = s_tiles[groups];
  const int n_kb = (p.k + kTcK - 1) / kTcK;
  volatile int* abort = &s_abort;
  TileWalk walk{s_rows, s_tiles, groups, ft, BN};

  if (warp == 0) {
    if (lane == 0) {
      uint32_t it = 0;
      bool ok = true;
      for (int i = blockIdx.x; ok && i < n_tiles; i += gridDim.x) {
        const TileWalk::Tile t = walk.at(i);
        const int wrow = t.group * (GATED ? 2 : 1) * p.n + t.feature0;
        for (int kb = 0; kb < n_kb; ++kb, ++it) {
          const uint32_t s = it % S::kStages, ph = (it / S::kStages) & 1u;
          if (!mbar_wait(&empty[s], ph ^ 1u, abort)) {
            set_status(p.status, ST_WAIT_EMPTY_TIMEOUT);
            ok = false;
            break;
          }
          uint8_t* st = ring + s * S::kStageBytes;
          mbar_expect_tx(&full[s], S::kStageBytes);
          tma_load_2d(st, &wmap, kb * kTcK, wrow, &full[s]);
          if (GATED) tma_load_2d(st + S::kWBytes, &wmap, kb * kTcK, wrow + p.n, &full[s]);
          tma_load_2d(st + (GATED ? 2 : 1) * S::kWBytes, &xmap, kb * kTcK, t.row0, &full[s]);
        }
      }
      if (!ok) *abort = 1;
      // copies still in flight must land before this CTA's shared memory goes away
      for (uint32_t j = it > S::kStages ? it - S::kStages : 0; j < it; ++j) mbar_wait(&full[j % S::kStages], (j / S::kStages) & 1u);
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = umma_idesc_bf16(128, BN);
      uint32_t it = 0, n_done = 0;
      bool ok = true;
      for (int i = blockIdx.x; ok && i < n_tiles; i += gridDim.x, ++n_done) {
        const uint32_t buf = n_done & 1u, aph = (n_done >> 1) & 1u;
        if (!mbar_wait(&acc_empty[buf], aph ^ 1u, abort)) {
          set_status(p.status, ST_WAIT_EMPTY_TIMEOUT);
          ok = false;
          break;
        }
        tc_fence_after();
        const uint32_t d = tmem + buf * S::kAccCols;
        for (int kb = 0; kb < n_kb; ++kb, ++it) {
          const uint32_t s = it % S::kStages, ph = (it / S::kStages) & 1u;
          if (!mbar_wait(&full[s], ph, abort)) {
            set_status(p.status, ST_WAIT_FULL_TIMEOUT);
            ok = false;
            break;
          }
          tc_fence_after();
          const uint32_t base = smem_u32(ring + s * S::kStageBytes);
          const uint64_t wd = umma_desc_sw128(base), ud = umma_desc_sw128(base + S::kWBytes);
          const uint64_t xd = umma_desc_sw128(base + (GATED ? 2 : 1) * S::kWBytes);
#pragma unroll
          for (int q = 0; q < kTcK / 16; ++q) {  // 32 bytes along K per instruction
            umma_bf16(d, wd + 2 * q, xd + 2 * q, idesc, (kb | q) != 0);
            if (GATED) umma_bf16(d + BN, ud + 2 * q, xd + 2 * q, idesc, (kb | q) != 0);
          }
          umma_commit(&empty[s]);
        }
        if (ok) umma_commit(&acc_full[buf]);
      }
      if (!ok) *abort = 1;
      umma_commit(&drain);  // products still running read shared memory and write TMEM
      mbar_wait(&drain, 0);
    }
  } else {
    const int quad = warp & 3;  // TMEM lanes this warp may read
    constexpr int kCols = BN / (kTcEpiWarps / 4);
    const int c0 = (warp - 2) / 4 * kCols;  // its columns
    const uint32_t lane_off = static_cast<uint32_t>(quad * 32) << 16;
    const bool pairs = p.out_bf16 && (p.n & 1) == 0 && (p.ldo & 1) == 0;
    const bool eights = p.out_bf16 && (p.n & 7) == 0 && (p.ldo & 7) == 0 && (reinterpret_cast<uintptr_t>(p.out) & 15) == 0;
    uint32_t n_done = 0;
    for (int i = blockIdx.x; i < n_tiles; i += gridDim.x, ++n_done) {
      const TileWalk::Tile t = walk.at(i);
      const uint32_t buf = n_done & 1u, aph = (n_done >> 1) & 1u;
      const bool ok = mbar_wait(&acc_full[buf], aph, abort);
      if (__any_sync(0xffffffffu, !ok)) {  // warp-uniform: tcgen05.ld needs every lane
        if (!ok) set_status(p.status, ST_WAIT_FULL_TIMEOUT);
        *abort = 1;
        break;
      }
      tc_fence_after();
      const int f = t.feature0 + quad * 32 + lane;
      const bool f_ok = f < p.n;
      const float bias = p.bias != nullptr && f_ok ? p.bias[f] : 0.f;
      const uint32_t acc = tmem + buf * S::kAccCols + lane_off;
      for (int c = c0; c < c0 + kCols && t.row0 + c < t.row1; c += 16) {
        float v[16];
        uint32_t r[16];
        tmem_ld16(acc + c, r);
        if (GATED) {
          uint32_t u[16];
          tmem_ld16(acc + BN + c, u);
          tmem_ld16_wait(r);
          tmem_ld16_wait(u);
#pragma unroll
          for (int j = 0; j < 16; ++j) v[j] = clamped_gate(__uint_as_float(r[j]), __uint_as_float(u[j]), p.limit, p.alpha);
        } else {
          tmem_ld16_wait(r);
#pragma unroll
          for (int j = 0; j < 16; ++j) v[j] = __uint_as_float(r[j]) + bias;
        }
        const int left = t.row1 - (t.row0 + c);
        if (!p.out_bf16) {
          float* o = reinterpret_cast<float*>(p.out) + static_cast<long long>(t.row0 + c) * p.ldo + f;
#pragma unroll
          for (int j = 0; j < 16; ++j)
            if (f_ok && j < left) o[j * p.ldo] = v[j];
        } else if (eights) {
          // eight lanes turn their eight features of eight tokens over: a lane stores eight features of one token
          __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(p.out) + static_cast<long long>(t.row0 + c) * p.ldo + (f & ~7);
#pragma unroll
          for (int j = 0; j < 16; j += 8) {
            const uint4 w = turn_eight(v + j, lane);
            const int jj = j + (lane & 7);
            if (f_ok && jj < left) *reinterpret_cast<uint4*>(o + jj * p.ldo) = w;
          }
        } else if (pairs) {
          // neighbouring lanes exchange one value, so that a lane stores two features of one token
          __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(p.out) + static_cast<long long>(t.row0 + c) * p.ldo + (f & ~1);
          const bool odd = lane & 1;
#pragma unroll
          for (int j = 0; j < 16; j += 2) {
            const float got = __shfl_xor_sync(0xffffffffu, odd ? v[j] : v[j + 1], 1);
            const int jj = j + (odd ? 1 : 0);
            const uint32_t w = odd ? pack_bf16x2(got, v[j + 1]) : pack_bf16x2(v[j], got);
            if (f_ok && jj < left) *reinterpret_cast<uint32_t*>(o + jj * p.ldo) = w;
          }
        } else {
          __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(p.out) + static_cast<long long>(t.row0 + c) * p.ldo + f;
#pragma unroll
          for (int j = 0; j < 16; ++j)
            if (f_ok && j < left) o[j * p.ldo] = f2bf(v[j]);
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&acc_empty[buf]);
    }
  }
  __syncwarp();
  tc_fence_before();
  __syncthreads();
  if (warp == 2) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(S::kTmemCols) : "memory");
  }
}

// ------------------------------------------------------------------ f32
constexpr int kF32Threads = 256, kF32Tile = 64, kF32K = 16;

template <bool GATED>
__global__ void __launch_bounds__(kF32Threads) gemm_f32_kernel(const GemmRowsParams p) {
  __shared__ float ws[GATED ? 2 : 1][kF32K][kF32Tile + 4], xs[kF32K][kF32Tile + 4];
  __shared__ int s_rows[kMaxGroups + 1], s_tiles[kMaxGroups + 1];
  pdl_launch_dependents();
  pdl_wait();
  constexpr int kW = GATED ? 2 : 1;
  // tiles of 128 features are walked as two halves of 64
  const int ft = (p.n + 127) / 128;
  tile_prefix(p, kF32Tile, ft, s_rows, s_tiles);
  const int groups = p.n_groups > 0 ? p.n_groups : 1;
  const int n_tiles = s_tiles[groups];
  TileWalk walk{s_rows, s_tiles, groups, ft, kF32Tile};
  const int tn = threadIdx.x & 15, tt = threadIdx.x >> 4;  // features tn + 16 i, tokens tt + 16 i
  for (int i2 = blockIdx.x; i2 < 2 * n_tiles; i2 += gridDim.x) {
    const TileWalk::Tile t = walk.at(i2 >> 1);
    const int f0 = t.feature0 + (i2 & 1) * kF32Tile;
    if (f0 >= p.n) continue;  // uniform over the CTA
    float acc[kW][4][4];
#pragma unroll
    for (int h = 0; h < kW; ++h)
#pragma unroll
      for (int a = 0; a < 4; ++a)
#pragma unroll
        for (int b = 0; b < 4; ++b) acc[h][a][b] = 0.f;
    for (int k0 = 0; k0 < p.k; k0 += kF32K) {
      for (int e = threadIdx.x; e < kF32Tile * kF32K; e += kF32Threads) {
        const int r = e / kF32K, c = e % kF32K;
        const bool kin = k0 + c < p.k;
#pragma unroll
        for (int h = 0; h < kW; ++h) {
          const long long row = (static_cast<long long>(t.group) * kW + h) * p.n + f0 + r;
          ws[h][c][r] = kin && f0 + r < p.n ? bf2f(p.w[row * p.ldw + k0 + c]) : 0.f;
        }
        xs[c][r] = kin && t.row0 + r < t.row1 ? p.x[static_cast<long long>(t.row0 + r) * p.ldx + k0 + c] : 0.f;
      }
      __syncthreads();
#pragma unroll
      for (int c = 0; c < kF32K; ++c) {
        float xv[4];
#pragma unroll
        for (int b = 0; b < 4; ++b) xv[b] = xs[c][tt + 16 * b];
#pragma unroll
        for (int h = 0; h < kW; ++h)
#pragma unroll
          for (int a = 0; a < 4; ++a) {
            const float wv = ws[h][c][tn + 16 * a];
#pragma unroll
            for (int b = 0; b < 4; ++b) acc[h][a][b] += wv * xv[b];
          }
      }
      __syncthreads();
    }
#pragma unroll
    for (int a = 0; a < 4; ++a)
#pragma unroll
      for (int b = 0; b < 4; ++b) {
        const int f = f0 + tn + 16 * a, r = t.row0 + tt + 16 * b;
        if (f < p.n && r < t.row1) {
          const float v = GATED ? clamped_gate(acc[0][a][b], acc[kW - 1][a][b], p.limit, p.alpha)
                                : acc[0][a][b] + (p.bias != nullptr ? p.bias[f] : 0.f);
          reinterpret_cast<float*>(p.out)[static_cast<long long>(r) * p.ldo + f] = v;
        }
      }
  }
}

}  // namespace tb
