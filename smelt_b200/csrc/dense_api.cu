// Typed launchers of the dense-weight decoders' kernels.
#include "dense.h"
#include "runtime.h"
#include "stack.h"

using namespace smelt;

namespace {

smelt_status enter(smelt_cuda_ctx* ctx, Launch* l, uint32_t position = 0) {
    if (!ctx) return SMELT_ERR_BAD_ARGUMENT;
    if (cudaSetDevice(ctx->device) != cudaSuccess) return fail(ctx, SMELT_ERR_CUDA, "cudaSetDevice");
    l->stream = ctx->stream;
    l->pdl = ctx->capturing && ctx->pdl;
    l->position = position;
    return SMELT_OK;
}

bool known(int precision) { return precision == SMELT_DENSE_BF16 || precision == SMELT_DENSE_F32; }

smelt_status window_args(smelt_cuda_ctx* ctx, const smelt_window_desc* d, int precision, int m, WindowArgs* a) {
    if (!d || !known(precision) || m <= 0 || d->heads <= 0 || d->kv_heads <= 0 || d->heads % d->kv_heads || d->dim <= 0 || d->vdim <= 0 || d->window == 0 || d->pool == 0 || d->ring == 0)
        return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "window attention: bad geometry or precision");
    if ((uint64_t)d->ring + 1 < (uint64_t)(d->window > d->pool ? d->window : d->pool) + (uint64_t)m)
        return fail(ctx, SMELT_ERR_OUT_OF_RANGE, "window attention: the ring is too short for the window and the chunk");
    *a = {};
    a->heads = d->heads; a->kv_heads = d->kv_heads; a->dim = d->dim; a->vdim = d->vdim;
    a->kp = window_padded(d->dim); a->vp = window_padded(d->vdim);
    a->window = d->window; a->pool = d->pool; a->ring = d->ring; a->blocks = d->blocks;
    a->scale = d->scale; a->softcap = d->softcap; a->eps = d->eps; a->m = m; a->sm_count = ctx->sm_count;
    return SMELT_OK;
}

}  // namespace

extern "C" {

smelt_status smelt_cuda_dense_gemm(smelt_cuda_ctx* ctx, int precision, int mode, const void* w, const void* x, void* y0, void* y1, int rows, int cols, int m, int split, int ld0,
                                   int ld1, float rising, float falling) {
    Launch l;
    smelt_status s = enter(ctx, &l);
    if (s) return s;
    if (!known(precision) || mode < 0 || mode > 2 || !w || !x || !y0 || (split < rows && !y1) || rows <= 0 || cols <= 0 || cols % 64 || m <= 0 || split < 0 || split > rows)
        return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "dense gemm: bad arguments (cols a multiple of 64)");
    DenseGemmArgs a = {};
    a.w = (const bf16*)w; a.x = x; a.rows = rows; a.cols = cols; a.m = m;
    a.out = {y0, y1, ld0, ld1, split, rising, falling};
    a.sm_count = ctx->sm_count; a.err = ctx->err_dev;
    a.part_scratch = ctx->qmm_scratch; a.part_scratch_bytes = ctx->qmm_scratch_bytes; a.part_counters = ctx->qmm_counters;
    return check_cuda(ctx, launch_dense_gemm(l, (DenseType)precision, mode, a), "dense gemm");
}

smelt_status smelt_cuda_dense_gemm_ex(smelt_cuda_ctx* ctx, int precision, int mode, const void* w, const void* x, const void* bias, void* y0, void* y1, int rows, int cols, int m,
                                      int split, int ld0, int ld1, int act, int group_rows) {
    Launch l;
    smelt_status s = enter(ctx, &l);
    if (s) return s;
    if (!known(precision) || (mode != kDenseStoreF32 && mode != kDenseStoreAct && mode != kDenseStoreMixed) || !w || !x || (split > 0 && !y0) || (split < rows && !y1) || rows <= 0 || cols <= 0 ||
        cols % 64 || m <= 0 || split < 0 || split > rows || act < 0 || act > 3 || group_rows < 0 || group_rows % 128 || (group_rows && rows <= (kMixes - 1) * group_rows))
        return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "dense gemm: bad arguments (cols a multiple of 64, groups of 128)");
    DenseGemmArgs a = {};
    a.w = (const bf16*)w; a.x = x; a.rows = rows; a.cols = cols; a.m = m;
    a.out = {y0, y1, ld0, ld1, split, 0.f, 0.f, act, (const bf16*)bias};
    a.group_rows = group_rows; a.x_group = group_rows ? m : 0; a.groups = group_rows ? kMixes : 0;
    a.sm_count = ctx->sm_count; a.err = ctx->err_dev;
    a.part_scratch = ctx->qmm_scratch; a.part_scratch_bytes = ctx->qmm_scratch_bytes; a.part_counters = ctx->qmm_counters;
    return check_cuda(ctx, launch_dense_gemm(l, (DenseType)precision, mode, a), "dense gemm");
}

smelt_status smelt_cuda_dense_matvec(smelt_cuda_ctx* ctx, int mode, const void* w, const void* xa, const void* xb, int ka, void* y0, void* y1, int rows, int cols, int split,
                                     int norm_width, float gain, float eps, float rising, float falling) {
    Launch l;
    smelt_status s = enter(ctx, &l);
    if (s) return s;
    if (mode < 0 || mode > 1 || !w || !xa || !y0 || (split < rows && !y1) || rows <= 0 || cols <= 0 || cols % 64 || split < 0 || split > rows || (xb && (ka <= 0 || ka % 4 || ka >= cols)))
        return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "dense matvec: bad arguments (cols a multiple of 64)");
    DenseMatvecArgs a = {};
    a.w = (const bf16*)w; a.xa = (const float*)xa; a.xb = (const float*)xb; a.ka = xb ? ka : cols; a.rows = rows; a.cols = cols;
    a.norm = norm_width > 0; a.width = norm_width; a.gain = gain; a.eps = eps;
    a.out = {y0, y1, 0, 0, split, rising, falling};
    a.sm_count = ctx->sm_count;
    return check_cuda(ctx, launch_dense_matvec(l, mode, a), "dense matvec");
}

smelt_status smelt_cuda_embed_positions(smelt_cuda_ctx* ctx, const void* table, const void* tokens, const void* positions, void* x, void* x0, int width, int ld, int m, uint32_t vocab,
                                        uint32_t max_positions, float scale, uint32_t position) {
    Launch l;
    smelt_status s = enter(ctx, &l, position);
    if (s) return s;
    if (!table || !tokens || !positions || !x || !x0 || (uint64_t)position + (uint64_t)m > max_positions) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "embed positions: bad arguments");
    return check_cuda(ctx, launch_embed_positions(l, (const bf16*)table, (const int32_t*)tokens, (const bf16*)positions, (float*)x, (float*)x0, width, ld, m, vocab, max_positions, scale), "embed positions");
}

smelt_status smelt_cuda_scalar_norm_rows(smelt_cuda_ctx* ctx, int precision, const void* x, const void* rows, void* out, int width, int ld, int m, float gain, float eps) {
    Launch l;
    smelt_status s = enter(ctx, &l);
    if (s) return s;
    if (!known(precision) || !x || !out) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "scalar norm: bad arguments");
    return check_cuda(ctx, launch_scalar_norm_rows(l, (DenseType)precision, (const float*)x, (const int32_t*)rows, out, width, ld, m, gain, eps), "scalar norm");
}

smelt_status smelt_cuda_pair_rows(smelt_cuda_ctx* ctx, int precision, const void* x, const void* x0, void* out, int ld, int m) {
    Launch l;
    smelt_status s = enter(ctx, &l);
    if (s) return s;
    if (!known(precision) || !x || !x0 || !out) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "pair rows: bad arguments");
    return check_cuda(ctx, launch_pair_rows(l, (DenseType)precision, (const float*)x, (const float*)x0, out, ld, m), "pair rows");
}

smelt_status smelt_cuda_window_append(smelt_cuda_ctx* ctx, int precision, const smelt_window_desc* d, const void* u, const void* q_norm, const void* k_norm, void* k_cache, void* v_cache,
                                      void* q, int m, uint32_t position) {
    Launch l;
    WindowArgs a;
    smelt_status s = enter(ctx, &l, position);
    if (!s) s = window_args(ctx, d, precision, m, &a);
    if (s) return s;
    if (!u || !q_norm || !k_norm || !k_cache || !v_cache || !q) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "window append: null pointer");
    a.u = u; a.q_norm = (const bf16*)q_norm; a.k_norm = (const bf16*)k_norm; a.k_cache = k_cache; a.v_cache = v_cache; a.q = q;
    return check_cuda(ctx, launch_window_append(l, (DenseType)precision, a), "window append");
}

smelt_status smelt_cuda_window_pool(smelt_cuda_ctx* ctx, int precision, const smelt_window_desc* d, void* k_cache, void* v_cache, int m, uint32_t position) {
    Launch l;
    WindowArgs a;
    smelt_status s = enter(ctx, &l, position);
    if (!s) s = window_args(ctx, d, precision, m, &a);
    if (s) return s;
    if (!k_cache || !v_cache) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "window pool: null pointer");
    a.k_cache = k_cache; a.v_cache = v_cache;
    return check_cuda(ctx, launch_window_pool(l, (DenseType)precision, a), "window pool");
}

smelt_status smelt_cuda_window_attention(smelt_cuda_ctx* ctx, int precision, const smelt_window_desc* d, const void* q, void* k_cache, void* v_cache, void* z, int ldz, int m,
                                         uint32_t position) {
    Launch l;
    WindowArgs a;
    smelt_status s = enter(ctx, &l, position);
    if (!s) s = window_args(ctx, d, precision, m, &a);
    if (s) return s;
    if (!q || !k_cache || !v_cache || !z || ldz < d->heads * d->vdim || (ldz % 2 && d->vdim % 2 == 0)) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "window attention: null pointer or short output rows");
    a.q = const_cast<void*>(q); a.k_cache = k_cache; a.v_cache = v_cache; a.z = z; a.ldz = ldz;
    return check_cuda(ctx, launch_window_attention(l, (DenseType)precision, a), "window attention");
}

smelt_status smelt_cuda_window_decode(smelt_cuda_ctx* ctx, int precision, const smelt_window_desc* d, const void* u, const void* q_norm, const void* k_norm, void* k_cache, void* v_cache,
                                      void* q, void* z, uint32_t position) {
    Launch l;
    WindowArgs a;
    smelt_status s = enter(ctx, &l, position);
    if (!s) s = window_args(ctx, d, precision, 1, &a);
    if (s) return s;
    if (!u || !q_norm || !k_norm || !k_cache || !v_cache || !q || !z) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "window decode: null pointer");
    a.u = u; a.q_norm = (const bf16*)q_norm; a.k_norm = (const bf16*)k_norm; a.k_cache = k_cache; a.v_cache = v_cache; a.q = q; a.z = z; a.ldz = d->heads * d->vdim;
    int launches = 0;
    return check_cuda(ctx, launch_window_decode(l, (DenseType)precision, a, &launches), "window decode");
}

}  // extern "C"
