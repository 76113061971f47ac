// Typed launchers of the kernels of mixer / feed-forward stacks.
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

smelt_status latent_args(smelt_cuda_ctx* ctx, int precision, const smelt_latent_args* d, LatentArgs* a) {
    if (!d || !known(precision) || d->heads <= 0 || d->dim <= 0 || d->rot_dim <= 0 || d->vdim <= 0 || d->kv_rank <= 0 || d->q_rank <= 0 || d->window == 0 || d->ring == 0 || d->m <= 0 ||
        (d->decode && d->m != 1))
        return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "latent attention: bad geometry or precision");
    if ((uint64_t)d->ring + 1 < (uint64_t)d->window + (uint64_t)d->m) return fail(ctx, SMELT_ERR_OUT_OF_RANGE, "latent attention: the ring is too short for the window and the chunk");
    *a = {};
    a->heads = d->heads; a->dim = d->dim; a->rot = d->rot_dim; a->rot_dims = d->rot_dims; a->vdim = d->vdim; a->rank = d->kv_rank; a->q_rank = d->q_rank;
    a->dp = pad16(d->dim); a->rp = pad16(d->rot_dim); a->vp = latent_value_pad(d->vdim); a->kr = pad64(d->kv_rank); a->qp = pad64(d->q_rank);
    a->window = d->window; a->ring = d->ring; a->scale = d->scale; a->eps = d->eps; a->m = d->m; a->own = d->own; a->ldu = d->ldu; a->ldz = d->ldz; a->q_f32 = d->decode;
    a->u = (const float*)d->u; a->q_norm = (const bf16*)d->q_norm; a->kv_norm = (const bf16*)d->kv_norm; a->freq = (const double*)d->rot_freq; a->q = d->q; a->kv = (const bf16*)d->kv_proj;
    a->kv_rows = d->kv_rows; a->cq = d->query_latent; a->c_ring = d->latent_ring; a->rot_ring = d->rot_ring; a->qa = (float*)d->qa; a->part = (float*)d->sums; a->part_ml = (float2*)d->maxima;
    a->z = d->z; a->sm_count = ctx->sm_count;
    a->splits = latent_splits(*a, (DenseType)precision);
    return SMELT_OK;
}

smelt_status wkv_args(smelt_cuda_ctx* ctx, const smelt_wkv_args* d, WkvArgs* a) {
    if (!d || d->heads <= 0 || d->dim <= 0 || d->m <= 0 || d->ld <= 0) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "time mixing: bad geometry");
    *a = {};
    a->heads = d->heads; a->dim = d->dim; a->group = (d->heads * d->dim + 127) / 128 * 128; a->rank = d->rank; a->ld = d->ld; a->m = d->m; a->ldu = d->ldu; a->ldz = d->ldz; a->eps = d->eps;
    a->u = (const float*)d->u; a->w2 = (const bf16*)d->w2; a->w0 = (const bf16*)d->w0; a->bonus = (const bf16*)d->bonus; a->norm = (const bf16*)d->norm; a->decay = (const float*)d->decay;
    a->h = (const float*)d->h; a->mu = (const bf16*)d->mu; a->o = (const float*)d->o; a->state = (float*)d->state; a->before = (float*)d->before; a->out = d->out;
    a->sm_count = ctx->sm_count;
    return SMELT_OK;
}

}  // namespace

extern "C" {

smelt_status smelt_cuda_stack_matvec(smelt_cuda_ctx* ctx, const smelt_stack_matvec_args* d, uint32_t position) {
    Launch l;
    smelt_status s = enter(ctx, &l, position);
    if (s) return s;
    if (!d || !d->w || !d->x || !d->out || (d->input != SMELT_MATVEC_PLAIN && d->input < SMELT_MATVEC_EXPERTS_IN && !d->norm) || (d->y && (!d->post_norm || !d->x_out)) ||
        (d->input >= SMELT_MATVEC_EXPERTS_IN && !d->chosen) || (d->input == SMELT_MATVEC_EXPERTS_IN && !d->logits))
        return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "stack matvec: null pointer");
    StackMatvecArgs a = {};
    a.w = (const bf16*)d->w; a.rows = d->rows; a.cols = d->cols; a.width = d->width; a.x = (const float*)d->x; a.y = (const float*)d->y; a.post_w = (const bf16*)d->post_norm;
    a.norm_w = (const bf16*)d->norm; a.x_out = (float*)d->x_out; a.h_out = (float*)d->h_out; a.eps = d->eps; a.before = (const float*)d->before; a.mu = (const bf16*)d->mu;
    a.group_rows = d->group_rows; a.bias = (const bf16*)d->bias; a.act = d->act; a.out = (float*)d->out; a.logits = (const float*)d->logits; a.experts = d->experts; a.top = d->top;
    a.limit = d->limit; a.chosen = (int2*)d->chosen; a.sm_count = ctx->sm_count;
    return check_cuda(ctx, launch_stack_matvec(l, d->input, a), "stack matvec");
}

smelt_status smelt_cuda_embed_rows(smelt_cuda_ctx* ctx, const void* table, const void* tokens, void* x, int width, int ld, int m, uint32_t vocab, float scale) {
    Launch l;
    smelt_status s = enter(ctx, &l);
    if (s) return s;
    if (!table || !tokens || !x) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "embed rows: null pointer");
    return check_cuda(ctx, launch_embed_rows(l, (const bf16*)table, (const int32_t*)tokens, (float*)x, width, ld, m, vocab, scale), "embed rows");
}

smelt_status smelt_cuda_residual_norm_rows(smelt_cuda_ctx* ctx, int precision, void* x, const void* y, const void* post_norm, const void* norm, const void* rows, void* out, void* h_f32,
                                           int width, int ld, int m, float eps) {
    Launch l;
    smelt_status s = enter(ctx, &l);
    if (s) return s;
    if (!known(precision) || !x || !norm || !out || (y && !post_norm)) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "residual norm: bad arguments");
    ResidualNormArgs a = {};
    a.x = (float*)x; a.y = (const float*)y; a.post_w = (const bf16*)post_norm; a.norm_w = (const bf16*)norm; a.rows = (const int32_t*)rows; a.out = out; a.h_f32 = (float*)h_f32;
    a.width = width; a.ld = ld; a.m = m; a.eps = eps;
    return check_cuda(ctx, launch_residual_norm_rows(l, (DenseType)precision, a), "residual norm");
}

#define LATENT(needed)                                                                                        \
    Launch l;                                                                                                 \
    LatentArgs a;                                                                                             \
    smelt_status s = enter(ctx, &l, position);                                                                \
    if (!s) s = latent_args(ctx, precision, d, &a);                                                           \
    if (s) return s;                                                                                          \
    if (!(needed)) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "latent attention: null pointer");

smelt_status smelt_cuda_latent_append(smelt_cuda_ctx* ctx, int precision, const smelt_latent_args* d, uint32_t position) {
    LATENT(d->u && d->q_norm && d->query_latent && (!d->own || (d->kv_norm && d->latent_ring && d->rot_ring && d->rot_freq)));
    return check_cuda(ctx, launch_latent_append(l, (DenseType)precision, a), "latent append");
}
smelt_status smelt_cuda_latent_query(smelt_cuda_ctx* ctx, int precision, const smelt_latent_args* d, uint32_t position) {
    const bool append = d && d->decode && d->own;
    LATENT(d->q && d->kv_proj && d->qa && d->rot_freq && (!append || (d->u && d->kv_norm && d->latent_ring && d->rot_ring)));
    return check_cuda(ctx, launch_latent_query(l, (DenseType)precision, a, append), "latent query");
}
smelt_status smelt_cuda_latent_scores(smelt_cuda_ctx* ctx, int precision, const smelt_latent_args* d, uint32_t position) {
    LATENT(d->qa && d->latent_ring && d->rot_ring && d->sums && d->maxima);
    return check_cuda(ctx, launch_latent_scores(l, (DenseType)precision, a), "latent scores");
}
smelt_status smelt_cuda_latent_values(smelt_cuda_ctx* ctx, int precision, const smelt_latent_args* d, uint32_t position) {
    LATENT(d->sums && d->maxima && d->kv_proj && d->z);
    return check_cuda(ctx, launch_latent_values(l, (DenseType)precision, a), "latent values");
}
smelt_status smelt_cuda_latent_prefill(smelt_cuda_ctx* ctx, const smelt_latent_args* d, uint32_t position) {
    const int precision = SMELT_DENSE_BF16;
    LATENT(d->q && d->kv_rows && d->rot_ring && d->rot_freq && d->z);
    return check_cuda(ctx, launch_latent_prefill(l, a), "latent prefill");
}
#undef LATENT

int smelt_cuda_latent_splits(smelt_cuda_ctx* ctx, int precision, const smelt_latent_args* d) {
    LatentArgs a;
    return ctx && latent_args(ctx, precision, d, &a) == SMELT_OK ? a.splits : 0;
}

smelt_status smelt_cuda_wkv_decode(smelt_cuda_ctx* ctx, const smelt_wkv_args* d, uint32_t position) {
    Launch l;
    WkvArgs a;
    smelt_status s = enter(ctx, &l, position);
    if (!s) s = wkv_args(ctx, d, &a);
    if (s) return s;
    if (!d->u || !d->w2 || !d->w0 || !d->bonus || !d->norm || !d->state || !d->before || !d->h || !d->out) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "time mixing: null pointer");
    return check_cuda(ctx, launch_wkv_decode(l, a), "time mixing decode");
}
smelt_status smelt_cuda_wkv_shift(smelt_cuda_ctx* ctx, int precision, const smelt_wkv_args* d, uint32_t position) {
    Launch l;
    WkvArgs a;
    smelt_status s = enter(ctx, &l, position);
    if (!s) s = wkv_args(ctx, d, &a);
    if (s) return s;
    if (!known(precision) || !d->h || !d->before || !d->mu || !d->out) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "time mixing: null pointer");
    return check_cuda(ctx, launch_shift_mix_rows(l, (DenseType)precision, a), "token shift");
}
smelt_status smelt_cuda_wkv_prefill(smelt_cuda_ctx* ctx, const smelt_wkv_args* d, uint32_t position) {
    Launch l;
    WkvArgs a;
    smelt_status s = enter(ctx, &l, position);
    if (!s) s = wkv_args(ctx, d, &a);
    if (s) return s;
    if (!d->u || !d->decay || !d->bonus || !d->state || !d->before || !d->h || !d->out) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "time mixing: null pointer");
    return check_cuda(ctx, launch_wkv_prefill(l, a), "time mixing prefill");
}
smelt_status smelt_cuda_wkv_gate(smelt_cuda_ctx* ctx, int precision, const smelt_wkv_args* d) {
    Launch l;
    WkvArgs a;
    smelt_status s = enter(ctx, &l);
    if (!s) s = wkv_args(ctx, d, &a);
    if (s) return s;
    if (!known(precision) || !d->u || !d->o || !d->norm || !d->out) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "time mixing: null pointer");
    return check_cuda(ctx, launch_wkv_gate_rows(l, (DenseType)precision, a), "time mixing gate");
}

smelt_status smelt_cuda_moe_rows(smelt_cuda_ctx* ctx, int precision, const smelt_moe_args* d, int stages, int only) {
    Launch l;
    smelt_status s = enter(ctx, &l);
    if (s) return s;
    if (!d || !known(precision) || d->m <= 0 || d->experts <= 0 || d->top <= 0 || d->top > d->experts || d->top > kMaxTop || d->ff <= 0 || d->width <= 0 || !d->logits || !d->h || !d->up ||
        !d->down || !d->chosen || !d->place || !d->table || !d->permuted || !d->inner || !d->rows || !d->y)
        return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "experts: bad arguments");
    const DenseType type = (DenseType)precision;
    MoeArgs a = {};
    a.m = d->m; a.experts = d->experts; a.top = d->top; a.width = d->width; a.ld = pad64(d->width); a.tile = moe_tile(a.m, a.top, a.experts, type);
    a.logits = (const float*)d->logits; a.chosen = (int2*)d->chosen; a.place = (int32_t*)d->place; a.table = (int4*)d->table; a.h = d->h; a.permuted = d->permuted;
    a.y_rows = (const float*)d->rows; a.y = (float*)d->y;
    const int fp = pad64(d->ff);
    DenseGemmArgs g = {};
    g.m = a.m * a.top; g.table = a.table; g.experts = a.experts; g.tile = a.tile; g.max_entries = moe_max_entries(a.m, a.top, a.experts, a.tile); g.sm_count = ctx->sm_count; g.err = ctx->err_dev;
    auto step = [&](int i) { return only ? stages == i : i <= stages; };
    cudaError_t e = cudaSuccess;
    if (step(1)) e = launch_moe_route(l, a);
    if (e == cudaSuccess && step(2)) e = launch_moe_gather(l, type, a);
    if (e == cudaSuccess && step(3)) {
        g.w = (const bf16*)d->up; g.x = d->permuted; g.rows = 2 * fp; g.cols = a.ld;
        g.out = {d->inner, nullptr, fp, 0, g.rows, d->limit, 0.f, 0, nullptr};
        e = launch_dense_gemm(l, type, kDenseStoreGlu, g);
    }
    if (e == cudaSuccess && step(4)) {
        g.w = (const bf16*)d->down; g.x = d->inner; g.rows = d->width; g.cols = fp;
        g.out = {d->rows, nullptr, a.ld, 0, g.rows, 0.f, 0.f, 0, nullptr};
        e = launch_dense_gemm(l, type, kDenseStoreF32, g);
    }
    if (e == cudaSuccess && step(5)) e = launch_moe_combine(l, a);
    return check_cuda(ctx, e, "experts");
}

}  // extern "C"
