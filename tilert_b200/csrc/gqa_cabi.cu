// C ABI of the decoders with bf16 weight rows (grouped-query and latent attention, dense and routed feed-forwards):
// argument checks and kernel launches.
// Declarations: include/tilert_gqa.h.
#include "../../include/tilert_gqa.h"

#include <cuda.h>

#include <cmath>
#include <mutex>

#include "host_util.h"

#include "gemm_rows.cuh"
#include "latent_attention.cuh"
#include "latent_rows.cuh"
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
  const long long x_rows = p.n_groups > 0 && p.counts == nullptr ? static_cast<long long>(p.n_groups) * p.rows : p.rows;
  if (rc == TB_OK) rc = make_map(&xmap, p.x, x_rows, p.k, p.ldx, BN);
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
  TB_REQUIRE(ctx != nullptr && tokens != nullptr && table != nullptr && x != nullptr);
  TB_REQUIRE(rows >= 1 && dim >= 1 && vocab >= 1 && ld_table >= dim && ldx >= dim && (xh == nullptr || ldh >= dim));
  const EmbedNormParams p{tokens, reinterpret_cast<const __nv_bfloat16*>(table), ld_table, vocab, gain, eps, dim, x, ldx, xh, ldh,
                          ctx->status};
  if (f32) return go(embed_norm_kernel<float>, dim3(rows), dim3(kNormThreads), 0, stream, p);
  return go(embed_norm_kernel<__nv_bfloat16>, dim3(rows), dim3(kNormThreads), 0, stream, p);
}

extern "C" int tilert_gqa_residual_norm_op(TgContext* ctx, const float* y, long long ldy, const void* ye, long long lde,
                                           const int* slot_row, const float* slot_w, int top, const void* ysh, long long ldsh,
                                           const float* gain, const float* bias, const float* add, const float* gain2,
                                           const float* bias2, int centered, float eps, int rows, int dim, float* x, long long ldx,
                                           void* xh, long long ldh, int f32, void* stream) {
  TB_REQUIRE(ctx != nullptr && x != nullptr && rows >= 1 && dim >= 1 && ldx >= dim && (xh == nullptr || ldh >= dim));
  TB_REQUIRE((gain != nullptr) == (y != nullptr || ye != nullptr) && (bias == nullptr || gain != nullptr));
  TB_REQUIRE((gain2 == nullptr || xh != nullptr) && (bias2 == nullptr || gain2 != nullptr));
  TB_REQUIRE(y != nullptr ? ldy >= dim
                          : (ye == nullptr || (slot_row != nullptr && slot_w != nullptr && top >= 1 && stride_ok(lde, dim) && aligned16(ye) &&
                                               (ysh == nullptr || (stride_ok(ldsh, dim) && aligned16(ysh))))));
  const ResidualNormParams p{y,    ldy, ye,    lde,   slot_row, slot_w, top, ysh, ldsh, gain, bias,
                             add,  gain2, bias2, centered, eps, dim,    x,   ldx, xh,   ldh};
  const size_t smem = static_cast<size_t>(dim) * sizeof(float);
  if (f32) return go(residual_norm_kernel<float>, dim3(rows), dim3(kNormThreads), smem, stream, p);
  return go(residual_norm_kernel<__nv_bfloat16>, dim3(rows), dim3(kNormThreads), smem, stream, p);
}

extern "C" int tilert_gqa_gather_norm_op(TgContext* ctx, const float* x, long long ldx, const int* rows, int n, const float* gain,
                                         const float* bias, int centered, float eps, int dim, void* out, long long ldo, int f32, void* stream) {
  TB_REQUIRE(ctx != nullptr && x != nullptr && rows != nullptr && gain != nullptr && out != nullptr);
  TB_REQUIRE(n >= 1 && dim >= 1 && ldx >= dim && ldo >= dim);
  const GatherNormParams p{x, ldx, rows, gain, bias, centered, eps, dim, out, ldo};
  if (f32) return go(gather_norm_kernel<float>, dim3(n), dim3(kNormThreads), 0, stream, p);
  return go(gather_norm_kernel<__nv_bfloat16>, dim3(n), dim3(kNormThreads), 0, stream, p);
}

// ------------------------------------------------------------------------------- products
extern "C" int tilert_gqa_gemm_op(TgContext* ctx, const void* x, long long ldx, int rows, const void* w, long long ldw, int n, int k,
                                  int gated, float limit, float alpha, int n_groups, const int* counts, const float* bias, void* out,
                                  long long ldo, int out_f32, int f32, void* stream) {
  TB_REQUIRE(ctx != nullptr && x != nullptr && w != nullptr && out != nullptr);
  TB_REQUIRE(rows >= 1 && n >= 1 && k >= 1 && n_groups >= 0 && n_groups <= kMaxGroups);
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
    if (n_groups > 0) return bn == 64 || (counts != nullptr ? rows / n_groups : rows) >= bn * 3 / 4 ? 1.0 / bn : 1.0;
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

bool prefill_attn_fits(int dimp, int vdimp) { return vdimp <= 256 && attn_prefill_smem(dimp, vdimp) <= kMaxSmem; }

int run_prefill_attn(const AttnPrefillParams& p, void* stream) {
  const int group = p.s.heads / p.s.kv_heads, hpb = group < kFaMaxHeads ? group : kFaMaxHeads, tpb = kFaRows / hpb;
  const dim3 grid((p.rows + tpb - 1) / tpb, p.s.kv_heads * ((group + hpb - 1) / hpb));
  if (p.s.vdimp <= 64) return launch_prefill_attn<4>(p, grid, stream);
  if (p.s.vdimp <= 128) return launch_prefill_attn<8>(p, grid, stream);
  return launch_prefill_attn<16>(p, grid, stream);
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
  if (!f32 && prefill_attn_fits(s.dimp, s.vdimp)) {
    AttnPrefillParams p{};
    p.s = s;
    p.pos = pos;
    p.rows = rows;
    p.q = reinterpret_cast<const __nv_bfloat16*>(q);
    p.k_cache = reinterpret_cast<const __nv_bfloat16*>(k_cache);
    p.v_cache = reinterpret_cast<const __nv_bfloat16*>(v_cache);
    p.k_ld = p.dim1 = s.dimp;
    p.v_ld = s.vdimp;
    p.k_head = static_cast<long long>(ring) * s.dimp;
    p.v_head = static_cast<long long>(ring) * s.vdimp;
    p.scale = scale;
    p.out = reinterpret_cast<__nv_bfloat16*>(out);
    p.ldo = ldo;
    return run_prefill_attn(p, stream);
  }
  AttnRowsParams a{};
  a.s = s;
  a.pos = pos;
  a.q = q;
  a.q_head = s.dimp;
  a.q_token = static_cast<long long>(heads) * s.dimp;
  a.k_cache = const_cast<void*>(k_cache);
  a.v_cache = const_cast<void*>(v_cache);
  a.v_ld = s.vdimp;
  a.rows = rows;
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
namespace {

int check_stage(const RvStage& s) {
  TB_REQUIRE(s.x != nullptr && s.k >= 1 && (s.y == nullptr) == (s.gain == nullptr) && (s.bias == nullptr || s.gain != nullptr));
  TB_REQUIRE((s.bias2 == nullptr || s.gain2 != nullptr) && (s.x_out == nullptr || (s.x_out != s.x && s.x_out != s.y)));
  TB_REQUIRE(aligned16(s.x) && aligned16(s.y) && aligned16(s.gain) && aligned16(s.bias) && aligned16(s.add) && aligned16(s.gain2) &&
             aligned16(s.bias2) && aligned16(s.x_out));
  return TB_OK;
}

}  // namespace

extern "C" int tilert_gqa_vec_dense_op(TgContext* ctx, const float* x, const float* y, const float* gain, const float* norm_bias,
                                       const float* add, const float* gain2, const float* norm_bias2, int centered, float eps,
                                       float* x_out, const void* w, long long ldw, const float* bias, int n, int k, float* out,
                                       void* stream) {
  const RvStage in{x, y, gain, norm_bias, add, gain2, norm_bias2, x_out, eps, centered, k};
  const int rc = check_stage(in);
  if (rc != TB_OK) return rc;
  TB_REQUIRE(ctx != nullptr && w != nullptr && out != nullptr && n >= 1 && stride_ok(ldw, k) && aligned16(w));
  const RvDenseParams p{in, reinterpret_cast<const __nv_bfloat16*>(w), ldw, bias, n, out};
  const int grid = n < ctx->num_sms ? n : ctx->num_sms;
  return go(rv_dense_kernel, dim3(grid), dim3(kRvThreads), kRvPartBytes + rv_vec_bytes(pad_to(k, 8)), stream, p);
}

extern "C" int tilert_gqa_vec_gated_op(TgContext* ctx, const float* x, const float* y, const float* gain, const float* norm_bias,
                                       const float* add, const float* gain2, const float* norm_bias2, int centered, float eps,
                                       float* x_out, const void* w, long long ldw, int n, int k, float limit, float alpha, float* out,
                                       void* stream) {
  const RvStage in{x, y, gain, norm_bias, add, gain2, norm_bias2, x_out, eps, centered, k};
  const int rc = check_stage(in);
  if (rc != TB_OK) return rc;
  TB_REQUIRE(ctx != nullptr && w != nullptr && out != nullptr && n >= 1 && stride_ok(ldw, k) && aligned16(w));
  const RvGatedParams p{in, reinterpret_cast<const __nv_bfloat16*>(w), ldw, n, limit, alpha, out};
  const int grid = n < ctx->num_sms ? n : ctx->num_sms;
  return go(rv_gated_kernel, dim3(grid), dim3(kRvThreads), kRvPartBytes + rv_vec_bytes(pad_to(k, 8)), stream, p);
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
  a.v_ld = a.s.vdimp;
  a.rows = 1;
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

// ------------------------------------------------------------------------------- attention over a latent cache
namespace {

LatentRow latent_row(int rank, int rot) {
  const int rankp = pad_to(rank, 16);
  return {rank, rankp, rot, pad_to(rankp + rot, 32)};
}
int check_latent(const LatentRow& r, int heads, int ring) {
  TB_REQUIRE(r.rank >= 1 && r.rank <= 2048 && r.rot >= 1 && r.row <= 4096 && heads >= 1 && heads <= kMaxGroups && ring >= 1);
  return TB_OK;
}
int check_rotation(const Rotation& r, int rot) {
  TB_REQUIRE(r.table != nullptr && r.positions >= 1 && r.dims >= 0 && r.dims % 2 == 0 && r.dims <= rot);
  return TB_OK;
}

// Tiles of 16 query rows per CTA of the tensor-core kernel; 0: its tiles do not fit, the row kernel runs
int latent_tiles(int n_rows, const LatentRow& r) {
  if (r.rankp > 1024) return 0;
  if (n_rows > 16 && latent_attn_smem(2, r.row) <= kMaxSmem) return 2;
  return latent_attn_smem(1, r.row) <= kMaxSmem ? 1 : 0;
}

template <int MT>
int launch_latent(const LatentAttnParams& p, void* stream) {
  const dim3 grid(p.n_splits, (p.n_rows + 16 * MT - 1) / (16 * MT));
  const size_t smem = latent_attn_smem(MT, p.r.row);
  if (p.r.rankp <= 128) return go(latent_attn_kernel<MT, 1>, grid, dim3(kLaThreads), smem, stream, p);
  if (p.r.rankp <= 256) return go(latent_attn_kernel<MT, 2>, grid, dim3(kLaThreads), smem, stream, p);
  if (p.r.rankp <= 512) return go(latent_attn_kernel<MT, 4>, grid, dim3(kLaThreads), smem, stream, p);
  return go(latent_attn_kernel<MT, 8>, grid, dim3(kLaThreads), smem, stream, p);
}

}  // namespace

extern "C" int tilert_gqa_latent_row_len(int rank, int rot) { return latent_row(rank, rot).row; }

extern "C" int tilert_gqa_latent_blocks(int heads, int tokens, int rank, int rot, int f32) {
  const int mt = f32 ? 0 : latent_tiles(heads * tokens, latent_row(rank, rot));
  return mt > 0 ? (heads * tokens + 16 * mt - 1) / (16 * mt) : head_blocks(heads, 1) * tokens;
}

extern "C" int tilert_gqa_expanded_fits(int dim, int rot, int vdim) {
  return prefill_attn_fits(pad_to(dim, 16) + pad_to(rot, 16), pad_to(vdim, 16)) ? 1 : 0;
}

extern "C" int tilert_gqa_latent_tokens_op(TgContext* ctx, const float* z, long long ldz, int q_rank, int off_c, int off_r,
                                           const float* q_gain, const float* c_gain, float eps, int rows, int rank, int rot,
                                           const float* rope, int positions, int rope_dims, int interleaved, const int* pos, int ring,
                                           void* cq, long long ldq, void* cache, int f32, void* stream) {
  LatentTokensParams p{};
  p.r = latent_row(rank, rot);
  p.rope = {rope, positions, rope_dims, interleaved};
  int rc = check_latent(p.r, 1, ring);
  if (rc == TB_OK) rc = check_rotation(p.rope, rot);
  if (rc != TB_OK) return rc;
  TB_REQUIRE(ctx != nullptr && z != nullptr && q_gain != nullptr && c_gain != nullptr && pos != nullptr && cq != nullptr && cache != nullptr);
  TB_REQUIRE(rows >= 1 && rows <= ring && q_rank >= 1 && ldq >= q_rank && off_c >= 0 && off_r >= 0 && ldz >= off_c + rank && ldz >= off_r + rot);
  p.z = z;
  p.ldz = ldz;
  p.q_rank = q_rank;
  p.off_c = off_c;
  p.off_r = off_r;
  p.q_gain = q_gain;
  p.c_gain = c_gain;
  p.eps = eps;
  p.pos = pos;
  p.ring = ring;
  p.cq = cq;
  p.ldq = ldq;
  p.cache = cache;
  if (f32) return go(latent_tokens_kernel<float>, dim3(rows), dim3(256), 0, stream, p);
  return go(latent_tokens_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, stream, p);
}

extern "C" int tilert_gqa_latent_queries_op(TgContext* ctx, const float* q, long long ldq, int rows, int heads, int dim, int rot,
                                            const float* rope, int positions, int rope_dims, int interleaved, const int* pos, void* out,
                                            float* lat, int rank, int f32, void* stream) {
  LatentQueriesParams p{};
  p.rope = {rope, positions, rope_dims, interleaved};
  const int rc = check_rotation(p.rope, rot);
  if (rc != TB_OK) return rc;
  TB_REQUIRE(ctx != nullptr && q != nullptr && pos != nullptr && out != nullptr && rows >= 1 && heads >= 1 && dim >= 1 && rot >= 1);
  TB_REQUIRE(lat == nullptr || rank >= 1);
  p.q = q;
  p.ldq = ldq;
  p.heads = heads;
  p.dim = dim;
  p.dimp8 = pad_to(dim, 8);
  p.rot = rot;
  p.ldh = p.dimp8 + pad_to(rot, 8);
  TB_REQUIRE(ldq >= static_cast<long long>(heads) * p.ldh);
  p.pos = pos;
  p.rows = rows;
  p.out = out;
  p.wide = pad_to(dim, 16) + pad_to(rot, 16);
  p.lat = lat;
  if (lat != nullptr) {
    const LatentRow r = latent_row(rank, rot);
    p.off_rot = r.rankp;
    p.row = r.row;
  } else {
    p.off_rot = pad_to(dim, 16);
  }
  if (f32) return go(latent_queries_kernel<float>, dim3(rows), dim3(256), 0, stream, p);
  return go(latent_queries_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, stream, p);
}

extern "C" int tilert_gqa_latent_attn_op(TgContext* ctx, const float* q, const void* cache, int tokens, int heads, int rank, int rot,
                                         const int* pos, int window, int ring, float scale, int n_splits, float* part, int f32,
                                         void* stream) {
  const LatentRow r = latent_row(rank, rot);
  const int rc = check_latent(r, heads, ring);
  if (rc != TB_OK) return rc;
  TB_REQUIRE(ctx != nullptr && q != nullptr && cache != nullptr && pos != nullptr && part != nullptr && aligned16(q) && aligned16(cache) && aligned16(part));
  TB_REQUIRE(tokens >= 1 && tokens <= 32768 && window >= 0 && window + tokens - 1 <= ring && n_splits >= 1 && n_splits <= 1024);
  const int mt = f32 ? 0 : latent_tiles(heads * tokens, r);
  if (mt > 0) {
    LatentAttnParams p{};
    p.r = r;
    p.n_rows = heads * tokens;
    p.tokens = tokens;
    p.ring = ring;
    p.window = window;
    p.pos = pos;
    p.q = q;
    p.cache = reinterpret_cast<const __nv_bfloat16*>(cache);
    p.scale = scale;
    p.n_splits = n_splits;
    p.part = part;
    return mt == 2 ? launch_latent<2>(p, stream) : launch_latent<1>(p, stream);
  }
  AttnRowsParams a{};
  a.s = {heads, 1, r.row, r.rank, r.row, r.rankp, ring, window};
  a.pos = pos;
  a.q = q;
  a.q_head = static_cast<long long>(tokens) * r.row;
  a.q_token = r.row;
  a.k_cache = a.v_cache = const_cast<void*>(cache);
  a.v_ld = r.row;
  a.rows = tokens;
  a.scale = scale;
  a.n_splits = n_splits;
  a.part = part;
  a.parts_only = 1;
  const dim3 grid(n_splits, head_blocks(heads, 1), tokens);
  const size_t smem = attn_rows_smem(r.row, r.rankp);
  if (f32) return go(attn_rows_kernel<float, false, float>, grid, dim3(kAttnThreads), smem, stream, a);
  return go(attn_rows_kernel<__nv_bfloat16, false, float>, grid, dim3(kAttnThreads), smem, stream, a);
}

extern "C" int tilert_gqa_latent_merge_op(TgContext* ctx, const float* part, int tokens, int heads, int n_splits, int rank, int rot,
                                          const float* sink, void* out, long long ldo, int f32, void* stream) {
  const LatentRow r = latent_row(rank, rot);
  TB_REQUIRE(ctx != nullptr && part != nullptr && out != nullptr && tokens >= 1 && heads >= 1 && n_splits >= 1 && n_splits <= 1024 && ldo >= rank);
  const LatentMergeParams p{part, heads * tokens, tokens, n_splits, rank, r.rankp, sink, out, ldo};
  const size_t smem = sizeof(float) * n_splits;
  if (f32) return go(latent_merge_kernel<float>, dim3(heads * tokens), dim3(128), smem, stream, p);
  return go(latent_merge_kernel<__nv_bfloat16>, dim3(heads * tokens), dim3(128), smem, stream, p);
}

extern "C" int tilert_gqa_gate_heads_op(TgContext* ctx, const float* o, int ldv, int rows, int heads, int vdim, const float* gate,
                                        long long ldg, int per_head, void* out, long long ldo, int f32, void* stream) {
  TB_REQUIRE(ctx != nullptr && o != nullptr && out != nullptr && rows >= 1 && heads >= 1 && vdim >= 1 && ldv >= vdim);
  TB_REQUIRE(ldo >= static_cast<long long>(heads) * vdim && (gate == nullptr || ldg >= (per_head ? heads : heads * vdim)));
  const GateHeadsParams p{o, ldv, heads, vdim, rows, {gate, ldg, per_head}, out, ldo};
  if (f32) return go(gate_heads_kernel<float>, dim3(rows), dim3(256), 0, stream, p);
  return go(gate_heads_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, stream, p);
}

extern "C" int tilert_gqa_expanded_attn_op(TgContext* ctx, const void* q, const void* kv, const void* cache, int rows, int heads, int dim,
                                           int rot, int vdim, int rank, const int* pos, int window, int ring, float scale,
                                           const float* sink, const float* gate, long long ldg, int per_head, void* out, long long ldo,
                                           void* stream) {
  const LatentRow r = latent_row(rank, rot);
  const int rc = check_latent(r, heads, ring);
  if (rc != TB_OK) return rc;
  const int dimp = pad_to(dim, 16), rotp = pad_to(rot, 16), vdimp = pad_to(vdim, 16);
  TB_REQUIRE(ctx != nullptr && q != nullptr && kv != nullptr && cache != nullptr && pos != nullptr && out != nullptr && rows >= 1);
  TB_REQUIRE(aligned16(q) && aligned16(kv) && aligned16(cache) && dim >= 1 && vdim >= 1 && window >= 0 && window + rows - 1 <= ring);
  TB_REQUIRE(prefill_attn_fits(dimp + rotp, vdimp) && ldo >= static_cast<long long>(heads) * vdim && (vdim % 2 == 1 || ldo % 2 == 0));
  TB_REQUIRE(gate == nullptr || ldg >= (per_head ? heads : heads * vdim));
  AttnPrefillParams p{};
  p.s = {heads, heads, dim + rot, vdim, dimp + rotp, vdimp, ring, window};
  p.pos = pos;
  p.rows = rows;
  p.q = reinterpret_cast<const __nv_bfloat16*>(q);
  p.k_cache = reinterpret_cast<const __nv_bfloat16*>(kv);
  p.v_cache = p.k_cache + static_cast<long long>(heads) * dimp;
  p.k2 = reinterpret_cast<const __nv_bfloat16*>(cache) + r.rankp;
  p.k_head = p.dim1 = dimp;
  p.v_head = vdimp;
  p.k_ld = p.v_ld = static_cast<long long>(heads) * (dimp + vdimp);
  p.k2_ld = r.row;
  p.scale = scale;
  p.sink = sink;
  p.gate = {gate, ldg, gate != nullptr ? per_head : 0};
  p.out = reinterpret_cast<__nv_bfloat16*>(out);
  p.ldo = ldo;
  return run_prefill_attn(p, stream);
}

extern "C" int tilert_gqa_vec_absorb_op(TgContext* ctx, const float* q, int heads, int dim, int rank, int rot, const void* w, long long ldw,
                                        const float* rope, int positions, int rope_dims, int interleaved, const float* c, const float* kr,
                                        const float* c_gain, float eps, const int* pos, int ring, float* lat, void* cache, int f32,
                                        void* stream) {
  RvAbsorbParams p{};
  p.r = latent_row(rank, rot);
  p.rope = {rope, positions, rope_dims, interleaved};
  int rc = check_latent(p.r, heads, ring);
  if (rc == TB_OK) rc = check_rotation(p.rope, rot);
  if (rc != TB_OK) return rc;
  TB_REQUIRE(ctx != nullptr && q != nullptr && w != nullptr && c != nullptr && kr != nullptr && c_gain != nullptr && pos != nullptr && lat != nullptr && cache != nullptr);
  TB_REQUIRE(dim >= 1 && stride_ok(ldw, dim) && aligned16(w) && aligned16(q) && aligned16(lat) && aligned16(cache));
  p.q = q;
  p.heads = heads;
  p.dim = dim;
  p.dimp8 = pad_to(dim, 8);
  p.ldh = p.dimp8 + pad_to(rot, 8);
  p.w = reinterpret_cast<const __nv_bfloat16*>(w);
  p.ldw = ldw;
  p.c = c;
  p.kr = kr;
  p.c_gain = c_gain;
  p.eps = eps;
  p.pos = pos;
  p.ring = ring;
  p.lat = lat;
  p.cache = cache;
  const long long groups = static_cast<long long>(heads) * ((rank + 3) / 4);
  const int grid = groups < ctx->num_sms ? static_cast<int>(groups) : ctx->num_sms;
  const size_t smem = kRvPartBytes + sizeof(float) * rv_heads_span(heads, rank, grid) * rv_vec_stride(p.dimp8);
  if (f32) return go(rv_absorb_kernel<float>, dim3(grid), dim3(kRvThreads), smem, stream, p);
  return go(rv_absorb_kernel<__nv_bfloat16>, dim3(grid), dim3(kRvThreads), smem, stream, p);
}

extern "C" int tilert_gqa_vec_value_op(TgContext* ctx, const float* part, int heads, int vdim, int rank, int rot, int n_splits,
                                       const float* sink, const void* w, long long ldw, const float* gate, int per_head, float* out,
                                       void* stream) {
  const LatentRow r = latent_row(rank, rot);
  const int rc = check_latent(r, heads, 1);
  if (rc != TB_OK) return rc;
  TB_REQUIRE(ctx != nullptr && part != nullptr && w != nullptr && out != nullptr && vdim >= 1 && n_splits >= 1 && n_splits <= 1024);
  TB_REQUIRE(stride_ok(ldw, rank) && aligned16(w) && aligned16(part));
  const RvValueParams p{r, part, heads, vdim, n_splits, sink, reinterpret_cast<const __nv_bfloat16*>(w), ldw, {gate, 0, per_head}, out};
  const long long groups = static_cast<long long>(heads) * ((vdim + 3) / 4);
  const int grid = groups < ctx->num_sms ? static_cast<int>(groups) : ctx->num_sms;
  const size_t smem = kRvPartBytes + sizeof(float) * rv_heads_span(heads, vdim, grid) * (rv_vec_stride(pad_to(rank, 8)) + n_splits);
  return go(rv_value_kernel, dim3(grid), dim3(kRvThreads), smem, stream, p);
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
