// C ABI of the grouped-query attention / mixture-of-experts path: argument checks and kernel launches.
// Declarations: include/tilert_gqa.h.
#include "../../include/tilert_gqa.h"

#include <cuda.h>

#include <cmath>
#include <mutex>

#include "host_util.h"

#include "gemm_rows.cuh"
#include "moe_rows.cuh"
#include "norm_rows.cuh"
#include "rowvec.cuh"
#include "sampler.cuh"
#include "window_attention.cuh"

using namespace tb;

struct TgContext {
  int device = 0;
  int num_sms = 0;
  int* status = nullptr;
};

namespace {

constexpr size_t kMaxSmem = 227 * 1024;

cudaStream_t stream_of(void* s) { return static_cast<cudaStream_t>(s); }

template <typename... KArgs, typename... Args>
int go(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, void* stream, Args&&... args) {
  TB_REQUIRE(smem <= kMaxSmem);
  if (smem > 48 * 1024) TB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  TB_CUDA(launch(kernel, grid, block, smem, stream_of(stream), std::forward<Args>(args)...));
  ++g_launches;
  TB_CUDA(cudaGetLastError());
  return TB_OK;
}

bool aligned16(const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; }
bool stride_ok(long long ld, int n) { return ld % kActPad == 0 && ld >= n; }

using EncodeTiled = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                 const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                 CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

EncodeTiled encode_tiled() {
  static const EncodeTiled fn = [] {
    void* f = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPointByVersion("cuTensorMapEncodeTiled", &f, 12000, cudaEnableDefault, &q) != cudaSuccess ||
        q != cudaDriverEntryPointSuccess)
      f = nullptr;
    return reinterpret_cast<EncodeTiled>(f);
  }();
  return fn;
}

// bf16 matrix [rows, k] with row stride ld, read in boxes of box_rows x 64 (zero outside the matrix)
int make_map(CUtensorMap* map, const void* base, long long rows, int k, long long ld, int box_rows) {
  if (encode_tiled() == nullptr) return fail(TB_ESTATE, "cuTensorMapEncodeTiled is not available%s");
  const cuuint64_t dims[2] = {static_cast<cuuint64_t>(k), static_cast<cuuint64_t>(rows)};
  const cuuint64_t strides[1] = {static_cast<cuuint64_t>(ld) * 2};
  const cuuint32_t box[2] = {kTcK, static_cast<cuuint32_t>(box_rows)};
  const cuuint32_t steps[2] = {1, 1};
  const CUresult r = encode_tiled()(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, steps,
                                    CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                                    CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) return fail(TB_ECUDA, "cuTensorMapEncodeTiled failed%s");
  return TB_OK;
}

template <int BN, bool GATED>
int launch_tc(TgContext* ctx, const GemmRowsParams& p, long long w_rows, void* stream) {
  CUtensorMap wmap, xmap;
  int rc = make_map(&wmap, p.w, w_rows, p.k, p.ldw, 128);
  if (rc == TB_OK) rc = make_map(&xmap, p.x, p.rows, p.k, p.ldx, BN);
  if (rc != TB_OK) return rc;
  return go(gemm_tc_kernel<BN, GATED>, dim3(ctx->num_sms), dim3(kTcThreads), TcShape<BN, GATED>::kSmemBytes, stream, wmap, xmap, p);
}

QkvShape qkv_shape(int heads, int kv_heads, int dim, int vdim, int ring, int window) {
  return {heads, kv_heads, dim, vdim, pad_to(dim, 16), pad_to(vdim, 16), ring, window};
}

int check_qkv(const QkvShape& s) {
  TB_REQUIRE(s.heads >= 1 && s.kv_heads >= 1 && s.heads % s.kv_heads == 0 && s.dim >= 1 && s.vdim >= 1 && s.vdimp <= 2048);
  TB_REQUIRE(s.ring >= 1 && s.window >= 0 && s.window <= s.ring);
  return TB_OK;
}

}  // namespace

// ------------------------------------------------------------------------------- runtime
extern "C" const char* tilert_gqa_last_error(void) { return g_last_error.c_str(); }
extern "C" long long tilert_gqa_launch_count(void) { return g_launches; }
extern "C" int tilert_gqa_num_sms(TgContext* ctx) { return ctx != nullptr ? ctx->num_sms : 0; }

extern "C" int tilert_gqa_default_context(int device, TgContext** ctx_out) {
  static std::mutex mu;
  static TgContext* ctxs[64] = {};
  TB_REQUIRE(ctx_out != nullptr && device >= 0 && device < 64);
  std::lock_guard<std::mutex> lock(mu);
  if (ctxs[device] == nullptr) {
    TB_CUDA(cudaSetDevice(device));
    cudaDeviceProp prop;
    TB_CUDA(cudaGetDeviceProperties(&prop, device));
    if (prop.major < 10) return fail(TB_ESTATE, "this library is built for sm_100a only; device is %s", prop.name);
    int* status = nullptr;
    TB_CUDA(cudaMalloc(&status, 256));
    TB_CUDA(cudaMemset(status, 0, 256));
    TgContext* c = new TgContext();
    c->device = device;
    c->num_sms = prop.multiProcessorCount;
    c->status = status;
    ctxs[device] = c;
  }
  *ctx_out = ctxs[device];
  return TB_OK;
}

extern "C" int tilert_gqa_status(TgContext* ctx, int* status_out) {
  TB_REQUIRE(ctx != nullptr && status_out != nullptr);
  TB_CUDA(cudaSetDevice(ctx->device));
  TB_CUDA(cudaDeviceSynchronize());
  TB_CUDA(cudaMemcpy(status_out, ctx->status, sizeof(int), cudaMemcpyDeviceToHost));
  if (*status_out != 0) TB_CUDA(cudaMemset(ctx->status, 0, sizeof(int)));
  return TB_OK;
}

extern "C" int tilert_gqa_set_wait_budget(TgContext* ctx, long long cycles) {
  TB_REQUIRE(ctx != nullptr);
  TB_CUDA(cudaSetDevice(ctx->device));
  const long long v = cycles > 0 ? cycles : kDefaultWaitBudgetCycles;
  TB_CUDA(cudaMemcpyToSymbol(g_wait_budget_cycles, &v, sizeof(v)));
  return TB_OK;
}

// ------------------------------------------------------------------------------- norms
extern "C" int tilert_gqa_embed_norm_op(TgContext* ctx, const long long* tokens, const void* table, long long ld_table, int vocab,
                                        const float* gain, float eps, int rows, int dim, float* x, long long ldx, void* xh,
                                        long long ldh, int f32, void* stream) {
  TB_REQUIRE(ctx != nullptr && tokens != nullptr && table != nullptr && gain != nullptr && x != nullptr);
  TB_REQUIRE(rows >= 1 && dim >= 1 && vocab >= 1 && ld_table >= dim && ldx >= dim && (xh == nullptr || ldh >= dim));
  const EmbedNormParams p{tokens, reinterpret_cast<const __nv_bfloat16*>(table), ld_table, vocab, gain, eps, dim, x, ldx, xh, ldh,
                          ctx->status};
  if (f32) return go(embed_norm_kernel<float>, dim3(rows), dim3(kNormThreads), 0, stream, p);
  return go(embed_norm_kernel<__nv_bfloat16>, dim3(rows), dim3(kNormThreads), 0, stream, p);
}

extern "C" int tilert_gqa_residual_norm_op(TgContext* ctx, const float* y, long long ldy, const void* ye, long long lde,
                                           const int* slot_row, const float* slot_w, int top, const void* ysh, long long ldsh,
                                           const float* gain, float eps, int rows, int dim, float* x, long long ldx, void* xh,
                                           long long ldh, int f32, void* stream) {
  TB_REQUIRE(ctx != nullptr && gain != nullptr && x != nullptr && xh != nullptr && rows >= 1 && dim >= 1 && ldx >= dim && ldh >= dim);
  TB_REQUIRE(y != nullptr ? ldy >= dim
                          : (ye != nullptr && slot_row != nullptr && slot_w != nullptr && top >= 1 && stride_ok(lde, dim) && aligned16(ye) &&
                             (ysh == nullptr || (stride_ok(ldsh, dim) && aligned16(ysh)))));
  const ResidualNormParams p{y, ldy, ye, lde, slot_row, slot_w, top, ysh, ldsh, gain, eps, dim, x, ldx, xh, ldh};
  const size_t smem = static_cast<size_t>(dim) * sizeof(float);
  if (f32) return go(residual_norm_kernel<float>, dim3(rows), dim3(kNormThreads), smem, stream, p);
  return go(residual_norm_kernel<__nv_bfloat16>, dim3(rows), dim3(kNormThreads), smem, stream, p);
}

extern "C" int tilert_gqa_gather_norm_op(TgContext* ctx, const float* x, long long ldx, const int* rows, int n, const float* gain,
                                         float eps, int dim, void* out, long long ldo, int f32, void* stream) {
  TB_REQUIRE(ctx != nullptr && x != nullptr && rows != nullptr && gain != nullptr && out != nullptr);
  TB_REQUIRE(n >= 1 && dim >= 1 && ldx >= dim && ldo >= dim);
  const GatherNormParams p{x, ldx, rows, gain, eps, dim, out, ldo};
  if (f32) return go(gather_norm_kernel<float>, dim3(n), dim3(kNormThreads), 0, stream, p);
  return go(gather_norm_kernel<__nv_bfloat16>, dim3(n), dim3(kNormThreads), 0, stream, p);
}

// ------------------------------------------------------------------------------- products
extern "C" int tilert_gqa_gemm_op(TgContext* ctx, const void* x, long long ldx, int rows, const void* w, long long ldw, int n, int k,
                                  int gated, float limit, float alpha, int n_groups, const int* counts, const float* bias, void* out,
                                  long long ldo, int out_f32, int f32, void* stream) {
  TB_REQUIRE(ctx != nullptr && x != nullptr && w != nullptr && out != nullptr);
  TB_REQUIRE(rows >= 1 && n >= 1 && k >= 1 && n_groups >= 0 && n_groups <= kMaxGroups && (n_groups == 0 || counts != nullptr));
  TB_REQUIRE(stride_ok(ldx, k) && stride_ok(ldw, k) && ldo >= n && aligned16(x) && aligned16(w));
  TB_REQUIRE(bias == nullptr || (n_groups == 0 && !gated));
  const int per = gated ? 2 : 1;
  TB_REQUIRE(static_cast<long long>(n_groups > 0 ? n_groups : 1) * per * n < (1ll << 31) - 256);
  GemmRowsParams p{};
  p.n = n;
  p.k = k;
  p.rows = rows;
  p.n_groups = n_groups;
  p.counts = counts;
  p.limit = limit;
  p.alpha = alpha;
  p.bias = bias;
  p.out = out;
  p.ldo = ldo;
  p.out_bf16 = !(out_f32 || f32);
  p.status = ctx->status;
  p.w = reinterpret_cast<const __nv_bfloat16*>(w);
  p.ldw = ldw;
  p.x = reinterpret_cast<const float*>(x);
  p.ldx = ldx;
  if (f32) {
    const dim3 grid(ctx->num_sms * 4);
    return gated ? go(gemm_f32_kernel<true>, grid, dim3(kF32Threads), 0, stream, p)
                 : go(gemm_f32_kernel<false>, grid, dim3(kF32Threads), 0, stream, p);
  }
  const long long w_rows = static_cast<long long>(n_groups > 0 ? n_groups : 1) * per * n;
  const int ft = (n + 127) / 128;
  // Token tile.  One weight: waves of tiles over the SMs times the relative cost of a tile (a narrow tile moves more
  // bytes per product through the L2).  Groups: the widest tile that an average group nearly fills.
  auto cost = [&](int bn, double tile) {
    if (n_groups > 0) return bn == 64 || rows / n_groups >= bn * 3 / 4 ? 1.0 / bn : 1.0;
    return std::ceil(static_cast<double>(ft) * ((rows + bn - 1) / bn) / ctx->num_sms) * tile;
  };
  if (gated) return cost(128, 1.0) <= cost(64, 0.6) ? launch_tc<128, true>(ctx, p, w_rows, stream) : launch_tc<64, true>(ctx, p, w_rows, stream);
  const double c256 = cost(256, 1.0), c128 = cost(128, 0.75), c64 = cost(64, 0.55);
  if (c256 <= c128 && c256 <= c64) return launch_tc<256, false>(ctx, p, w_rows, stream);
  if (c128 <= c64) return launch_tc<128, false>(ctx, p, w_rows, stream);
  return launch_tc<64, false>(ctx, p, w_rows, stream);
}

// ------------------------------------------------------------------------------- attention of a portion
extern "C" int tilert_gqa_qkv_rows_op(TgContext* ctx, const float* qkv, long long ld, const float* q_gain, const float* k_gain, float eps,
                                      int v_mode, const float* lambda, float* v_first, int rows, int heads, int kv_heads, int dim,
                                      int vdim, const int* pos, void* q, void* k_cache, void* v_cache, int ring, int f32, void* stream) {
  QkvRowsParams a{};
  a.s = qkv_shape(heads, kv_heads, dim, vdim, ring, 0);
  const int rc = check_qkv(a.s);
  if (rc != TB_OK) return rc;
  TB_REQUIRE(ctx != nullptr && qkv != nullptr && q_gain != nullptr && k_gain != nullptr && pos != nullptr && q != nullptr &&
             k_cache != nullptr && v_cache != nullptr && rows >= 1 && rows <= ring);
  TB_REQUIRE(v_mode == VMIX_NONE || v_first != nullptr);
  TB_REQUIRE(v_mode != VMIX_BLEND || lambda != nullptr);
  a.p = {qkv, ld, q_gain, k_gain, eps, v_mode, lambda, v_first};
  a.pos = pos;
  a.q = q;
  a.k_cache = k_cache;
  a.v_cache = v_cache;
  if (f32) return go(qkv_rows_kernel<float>, dim3(rows), dim3(256), 0, stream, a);
  return go(qkv_rows_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, stream, a);
}

namespace {

int head_blocks(int heads, int kv_heads) {
  const int group = heads / kv_heads;
  return kv_heads * ((group + kAttnHeads - 1) / kAttnHeads);
}

template <int DV16>
int launch_prefill_attn(const AttnPrefillParams& p, dim3 grid, void* stream) {
  return go(attn_prefill_kernel<DV16>, grid, dim3(kFaThreads), attn_prefill_smem(p.s.dimp, p.s.vdimp), stream, p);
}

}  // namespace

extern "C" int tilert_gqa_head_blocks(int heads, int kv_heads) { return head_blocks(heads, kv_heads); }

extern "C" int tilert_gqa_attn_rows_op(TgContext* ctx, const void* q, const void* k_cache, const void* v_cache, int rows, int heads,
                                       int kv_heads, int dim, int vdim, const int* pos, int window, int ring, float scale, void* out,
                                       long long ldo, int f32, void* stream) {
  const QkvShape s = qkv_shape(heads, kv_heads, dim, vdim, ring, window);
  const int rc = check_qkv(s);
  if (rc != TB_OK) return rc;
  TB_REQUIRE(ctx != nullptr && q != nullptr && k_cache != nullptr && v_cache != nullptr && pos != nullptr && out != nullptr);
  TB_REQUIRE(rows >= 1 && ldo >= static_cast<long long>(heads) * vdim && window + rows - 1 <= ring);
  if (!f32 && s.vdimp <= 256 && attn_prefill_smem(s.dimp, s.vdimp) <= kMaxSmem) {
    AttnPrefillParams p{};
    p.s = s;
    p.pos = pos;
    p.rows = rows;
    p.q = reinterpret_cast<const __nv_bfloat16*>(q);
    p.k_cache = reinterpret_cast<const __nv_bfloat16*>(k_cache);
    p.v_cache = reinterpret_cast<const __nv_bfloat16*>(v_cache);
    p.scale = scale;
    p.out = reinterpret_cast<__nv_bfloat16*>(out);
    p.ldo = ldo;
    const int group = heads / kv_heads, hpb = group < kFaMaxHeads ? group : kFaMaxHeads, tpb = kFaRows / hpb;
    const dim3 grid((rows + tpb - 1) / tpb, kv_heads * ((group + hpb - 1) / hpb));
    if (s.vdimp <= 64) return launch_prefill_attn<4>(p, grid, stream);
    if (s.vdimp <= 128) return launch_prefill_attn<8>(p, grid, stream);
    return launch_prefill_attn<16>(p, grid, stream);
  }
  AttnRowsParams a{};
  a.s = s;
  a.pos = pos;
  a.q = q;
  a.k_cache = const_cast<void*>(k_cache);
  a.v_cache = const_cast<void*>(v_cache);
  a.scale = scale;
  a.n_splits = 1;
  a.out = out;
  a.ldo = ldo;
  const size_t smem = attn_rows_smem(s.dimp, s.vdimp);
  constexpr int kMaxZ = 32768;
  TB_REQUIRE(rows <= kMaxZ);
  const dim3 grid(1, head_blocks(heads, kv_heads), rows);
  if (f32) return go(attn_rows_kernel<float, false>, grid, dim3(kAttnThreads), smem, stream, a);
  return go(attn_rows_kernel<__nv_bfloat16, false>, grid, dim3(kAttnThreads), smem, stream, a);
}

// ------------------------------------------------------------------------------- routing of a portion
extern "C" int tilert_gqa_route_rows_op(TgContext* ctx, const float* logits, long long ldl, int rows, int n_experts, int top, int* ids,
                                        float* w, int* rank, int* counts, void* stream) {
  TB_REQUIRE(ctx != nullptr && logits != nullptr && ids != nullptr && w != nullptr && rank != nullptr && counts != nullptr);
  TB_REQUIRE(rows >= 1 && n_experts >= 1 && n_experts <= kMaxExperts && top >= 1 && top <= kMaxTop && top <= n_experts && ldl >= n_experts);
  TB_CUDA(cudaMemsetAsync(counts, 0, sizeof(int) * n_experts, stream_of(stream)));
  const RouteRowsParams p{logits, ldl, rows, n_experts, top, ids, w, rank, counts};
  return go(route_rows_kernel, dim3((rows + kRouteWarps - 1) / kRouteWarps), dim3(kRouteWarps * 32),
            sizeof(float) * kRouteWarps * n_experts, stream, p);
}

extern "C" int tilert_gqa_gather_rows_op(TgContext* ctx, const void* x, long long ldx, int rows, int dim, int n_experts, int top,
                                         const int* ids, const int* rank, const int* counts, void* xs, int* slot_row, int f32,
                                         void* stream) {
  TB_REQUIRE(ctx != nullptr && x != nullptr && ids != nullptr && rank != nullptr && counts != nullptr && xs != nullptr && slot_row != nullptr);
  TB_REQUIRE(rows >= 1 && dim >= 1 && stride_ok(ldx, dim) && aligned16(x) && aligned16(xs) && top >= 1 && top <= kMaxTop);
  const GatherRowsParams p{x, ldx, pad_to(dim, 8) / 8, top, n_experts, ids, rank, counts, xs, slot_row};
  if (f32) return go(gather_rows_kernel<float>, dim3(rows), dim3(256), 0, stream, p);
  return go(gather_rows_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, stream, p);
}

// ------------------------------------------------------------------------------- one-token step
extern "C" int tilert_gqa_vec_dense_op(TgContext* ctx, const float* x, const float* y, const float* gain, const float* gain2, float eps,
                                       float* x_out, const void* w, long long ldw, const float* bias, int n, int k, float* out,
                                       void* stream) {
  TB_REQUIRE(ctx != nullptr && x != nullptr && w != nullptr && out != nullptr && n >= 1 && k >= 1);
  TB_REQUIRE((y == nullptr) == (gain == nullptr) && (x_out == nullptr || (x_out != x && x_out != y)));
  TB_REQUIRE(stride_ok(ldw, k) && aligned16(w) && aligned16(x));
  const RvDenseParams p{{x, y, gain, gain2, x_out, eps, k}, reinterpret_cast<const __nv_bfloat16*>(w), ldw, bias, n, out};
  const int grid = n < ctx->num_sms ? n : ctx->num_sms;
  return go(rv_dense_kernel, dim3(grid), dim3(kRvThreads), kRvPartBytes + rv_vec_bytes(pad_to(k, 8)), stream, p);
}

extern "C" int tilert_gqa_vec_attn_op(TgContext* ctx, const float* qkv, const float* q_gain, const float* k_gain, float eps, int v_mode,
                                      const float* lambda, float* v_first, int heads, int kv_heads, int dim, int vdim, const int* pos,
                                      int window, int ring, float scale, void* k_cache, void* v_cache, int n_splits, float* part,
                                      int* counter, float* out, int f32, void* stream) {
  AttnRowsParams a{};
  a.s = qkv_shape(heads, kv_heads, dim, vdim, ring, window);
  const int rc = check_qkv(a.s);
  if (rc != TB_OK) return rc;
  TB_REQUIRE(ctx != nullptr && qkv != nullptr && q_gain != nullptr && k_gain != nullptr && pos != nullptr && k_cache != nullptr &&
             v_cache != nullptr && out != nullptr && n_splits >= 1 && n_splits <= 1024 && (n_splits == 1 || (part != nullptr && counter != nullptr)));
  TB_REQUIRE(v_mode == VMIX_NONE || v_first != nullptr);
  TB_REQUIRE(v_mode != VMIX_BLEND || lambda != nullptr);
  a.p = {qkv, 0, q_gain, k_gain, eps, v_mode, lambda, v_first};
  a.pos = pos;
  a.k_cache = k_cache;
  a.v_cache = v_cache;
  a.scale = scale;
  a.n_splits = n_splits;
  a.part = part;
  a.counter = reinterpret_cast<unsigned*>(counter);
  a.out = out;
  const dim3 grid(n_splits, head_blocks(heads, kv_heads), 1);
  const size_t smem = attn_rows_smem(a.s.dimp, a.s.vdimp);
  if (f32) return go(attn_rows_kernel<float, true>, grid, dim3(kAttnThreads), smem, stream, a);
  return go(attn_rows_kernel<__nv_bfloat16, true>, grid, dim3(kAttnThreads), smem, stream, a);
}

extern "C" int tilert_gqa_vec_gate_up_op(TgContext* ctx, const float* x, int dim, const float* logits, int n_experts, int top,
                                         const void* w, const void* w_sh, long long ldw, int ff, int ff_sh, float limit, float limit_sh,
                                         float alpha, float* hidden, int* slot_ids, float* slot_w, void* stream) {
  TB_REQUIRE(ctx != nullptr && x != nullptr && logits != nullptr && w != nullptr && hidden != nullptr && slot_ids != nullptr && slot_w != nullptr);
  TB_REQUIRE(dim >= 1 && n_experts >= 1 && n_experts <= kMaxExperts && top >= 1 && top <= kMaxTop && top <= n_experts);
  TB_REQUIRE(ff >= 1 && ff_sh >= 0 && (ff_sh == 0) == (w_sh == nullptr) && stride_ok(ldw, dim) && aligned16(w) && aligned16(w_sh) && aligned16(x));
  const RvGateUpParams p{x, dim, logits, n_experts, top, reinterpret_cast<const __nv_bfloat16*>(w),
                         reinterpret_cast<const __nv_bfloat16*>(w_sh), ldw, ff, ff_sh, limit, limit_sh, alpha, hidden, slot_ids, slot_w};
  const int feats = ff_sh + top * ff;
  const int grid = feats < ctx->num_sms ? feats : ctx->num_sms;
  const size_t smem = kRvPartBytes + rv_vec_bytes(pad_to(dim, 8)) + sizeof(float) * n_experts;
  return go(rv_gate_up_kernel, dim3(grid), dim3(kRvThreads), smem, stream, p);
}

extern "C" int tilert_gqa_vec_down_op(TgContext* ctx, const float* hidden, const int* slot_ids, const float* slot_w, int top,
                                      const void* w, const void* w_sh, int ff, int ff_sh, int dim, float* out, void* stream) {
  TB_REQUIRE(ctx != nullptr && hidden != nullptr && slot_ids != nullptr && slot_w != nullptr && w != nullptr && out != nullptr);
  TB_REQUIRE(top >= 1 && top <= kMaxTop && ff >= 1 && ff_sh >= 0 && (ff_sh == 0) == (w_sh == nullptr) && dim >= 1);
  TB_REQUIRE(aligned16(hidden) && aligned16(w) && aligned16(w_sh));
  const RvDownParams p{hidden, slot_ids, slot_w, top, reinterpret_cast<const __nv_bfloat16*>(w),
                       reinterpret_cast<const __nv_bfloat16*>(w_sh), ff, ff_sh, dim, out};
  const int kp = pad_to(ff_sh, 8) + top * pad_to(ff, 8);
  const int grid = dim < ctx->num_sms ? dim : ctx->num_sms;
  return go(rv_down_kernel, dim3(grid), dim3(kRvThreads), kRvPartBytes + rv_vec_bytes(kp) + sizeof(RvPiece) * (kp / 8), stream, p);
}

// ------------------------------------------------------------------------------- sampling
extern "C" int tilert_gqa_sample_op(TgContext* ctx, const float* logits, long long logits_stride, int tokens, int vocab,
                                    const float* config_dev, unsigned long long seed, unsigned long long* step_dev,
                                    unsigned long long step_value, int* token_out, float* token_logprob_out, float* topn_logprob_out,
                                    int* topn_index_out, void* stream) {
  TB_REQUIRE(ctx != nullptr && logits != nullptr && config_dev != nullptr && token_out != nullptr);
  TB_REQUIRE(tokens >= 1 && vocab >= 1 && logits_stride >= vocab);
  TB_REQUIRE((topn_logprob_out == nullptr) == (topn_index_out == nullptr));
  const SampleParams p{logits, logits_stride, vocab, config_dev, seed, step_dev, step_value, token_out, token_logprob_out,
                       topn_logprob_out, topn_index_out};
  return go(sample_kernel, dim3(tokens), dim3(kTopkThreads), 0, stream, p);
}
