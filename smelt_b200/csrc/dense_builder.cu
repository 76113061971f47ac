// Table builder for decoders with dense 16-bit weights and window + pooled-block attention
// (smelt_cuda_build_dense_decoder): slots, pipelines and the decode and prompt-chunk records.
//
// A layer is parallel: one norm feeds the mixer and the feed-forward, so its projections are two
// matrices, [q; k; v; up] and [o | down], and a decoded token takes three launches per layer run:
// norm + first matrix + xIELU, attention, second matrix + residual.
#include <algorithm>
#include <map>
#include <utility>
#include <vector>

#include "dense.h"
#include "record_writer.h"

using namespace smelt;

namespace {

enum DenseSlot : int {
    kDnEmbedding = 24,  // the embedding output, read again at the start of every loop pass
    kDnU = 20, kDnQ = 21, kDnZ = 23,
    kDnPfX = 2, kDnPfX0 = 3, kDnPfAct = 4, kDnPfU = 5, kDnPfQ = 6, kDnPfZ = 7,
};

struct Run {
    int layer;
    bool begins;  // first layer of a loop pass
};

std::vector<Run> layer_runs(const smelt_dense_desc* d) {
    std::vector<Run> runs;
    for (int l = 0; l < d->loop_start; ++l) runs.push_back({l, false});
    for (int t = 0; t < d->loop_times; ++t)
        for (int l = d->loop_start; l < d->loop_stop; ++l) runs.push_back({l, l == d->loop_start});
    for (int l = d->loop_stop; l < d->layers; ++l) runs.push_back({l, false});
    return runs;
}

constexpr int kArgmaxChunk = 2048;

int pad64(int n) { return (n + 63) / 64 * 64; }

struct LayerShape {
    int qkv, cols2, kp, vp;
    uint32_t ring, blocks;
};

LayerShape layer_shape(const smelt_dense_layer& w, uint32_t capacity, uint32_t max_chunk) {
    LayerShape s;
    s.qkv = w.heads * w.dim + w.kv_heads * (w.dim + w.vdim);
    s.cols2 = pad64(w.heads * w.vdim + w.ff);
    s.kp = window_padded(w.dim);
    s.vp = window_padded(w.vdim);
    s.ring = window_ring_rows(w.window, w.pool, max_chunk);
    s.blocks = capacity / w.pool;
    return s;
}

const char* validate(const smelt_dense_desc* d, const smelt_dense_layer* layers, uint32_t capacity, uint32_t max_chunk) {
    if (d->layers <= 0 || d->width <= 0 || d->vocab <= 0 || capacity == 0 || max_chunk == 0 || max_chunk > 1920) return "bad model size, capacity or chunk";
    if (d->loop_start < 0 || d->loop_stop < d->loop_start || d->loop_stop > d->layers || d->loop_times < 0) return "bad loop";
    if (d->precision != SMELT_DENSE_BF16 && d->precision != SMELT_DENSE_F32) return "unknown precision";
    if (capacity > d->max_positions) return "capacity beyond the position table";
    for (int l = 0; l < d->layers; ++l) {
        const smelt_dense_layer& w = layers[l];
        if (w.heads <= 0 || w.kv_heads <= 0 || w.heads % w.kv_heads || w.heads > 65535 || w.dim <= 0 || w.vdim <= 0 || w.dim > 65535 || w.vdim > 65535 || w.window == 0 || w.pool == 0 ||
            w.ff < 0)
            return "bad layer geometry";
    }
    return nullptr;
}

using SlotPlan = std::vector<std::pair<int, size_t>>;

// The slots one table binds, with their sizes.
SlotPlan slot_plan(const smelt_dense_desc* d, const smelt_dense_layer* layers, uint32_t capacity, uint32_t max_chunk, bool prefill) {
    const std::vector<Run> runs = layer_runs(d);
    const size_t Wp = pad64(d->width), V = d->vocab, T = max_chunk, es = d->precision == SMELT_DENSE_F32 ? 4 : 2, parts = (V + kArgmaxChunk - 1) / kArgmaxChunk;
    size_t u = 0, q = 0, z = 0;  // widest layer
    for (int l = 0; l < d->layers; ++l) {
        const LayerShape s = layer_shape(layers[l], capacity, max_chunk);
        u = std::max(u, (size_t)s.qkv);
        q = std::max(q, (size_t)layers[l].heads * s.kp);
        z = std::max(z, (size_t)s.cols2);
    }
    if (prefill)
        return {{kDnPfX, T * Wp * 4}, {kDnPfX0, T * Wp * 4}, {kDnPfAct, T * 2 * Wp * es}, {kDnPfU, T * u * es}, {kDnPfQ, T * q * es}, {kDnPfZ, T * z * es},
                {kLogits, T * V * 4}, {kArgmaxScratch, T * parts * 8}, {kArgmax, std::max<size_t>(T * 4, 8)}, {kTokenId, T * 4}, {kLogitRowsSlot, T * 4}};
    SlotPlan plan = {{kHiddenA, Wp * 4}, {kHiddenB, Wp * 4}, {kDnEmbedding, Wp * 4}, {kDnU, u * 4}, {kDnQ, q * 4}, {kDnZ, z * 4},
                     {kLogits, V * 4}, {kArgmax, 8}, {kTokenId, 4}, {kPosition, 8}, {kArgmaxScratch, parts * 8}};
    for (size_t r = 0; r < runs.size(); ++r) {
        const smelt_dense_layer& w = layers[runs[r].layer];
        const LayerShape sh = layer_shape(w, capacity, max_chunk);
        const size_t rows = (size_t)w.kv_heads * (sh.ring + sh.blocks);
        plan.push_back({kKvBase + 2 * (int)r, rows * sh.kp * es});
        plan.push_back({kKvBase + 2 * (int)r + 1, rows * sh.vp * es});
    }
    return plan;
}

smelt_status build(smelt_cuda_ctx* ctx, const smelt_dense_desc* d, const smelt_dense_layer* layers, uint32_t capacity, uint32_t max_chunk, bool prefill,
                   smelt_dispatch_record* records, size_t* n_records, std::vector<std::string>* names = nullptr) {
    if (!d || !layers || !n_records) return SMELT_ERR_BAD_ARGUMENT;
    if (const char* why = validate(d, layers, capacity, max_chunk)) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, std::string("build_dense: ") + why);
    const std::vector<Run> runs = layer_runs(d);
    const int W = d->width, Wp = pad64(W), V = d->vocab, chunk = kArgmaxChunk, parts = (V + chunk - 1) / chunk;
    const size_t es = d->precision == SMELT_DENSE_F32 ? 4 : 2;
    const std::string type = d->precision == SMELT_DENSE_F32 ? "_f32" : "_bf16";
    Emitter e{ctx, records, records ? *n_records : 0};
    if (ctx) {
        if (!records) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "build_dense: a context needs a record buffer (query the count with a null context)");
        if (cudaSetDevice(ctx->device) != cudaSuccess) return fail(ctx, SMELT_ERR_CUDA, "cudaSetDevice");
        if (!ctx->slots[kWeights].ptr) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "build_dense: upload the weights image to slot 30 first");
        if (kKvBase + 2 * runs.size() > ctx->slots.size()) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "build_dense: too many layer runs for the slot table");
        if (prefill && (!ctx->configured || !ctx->slots[kDnU].ptr)) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "build_dense: build the decode table first");
        for (auto& p : slot_plan(d, layers, capacity, max_chunk, prefill)) {
            smelt_status s = smelt_cuda_alloc_slot(ctx, p.first, p.second);
            if (s) return s;
        }
        if (prefill) {
            e.base = (int)ctx->pipelines.size();
        } else {
            smelt_cuda_runtime_config cfg = {};
            cfg.token_id_slot = kTokenId; cfg.position_slot = kPosition; cfg.weights_slot = kWeights; cfg.argmax_slot = kArgmax;
            cfg.cur_slot = kHiddenA; cfg.alt_slot = kHiddenB; cfg.cache_seq_capacity = capacity; cfg.context_limit = capacity;
            cfg.vocab_size = (uint32_t)V; cfg.batch = 1;
            smelt_status s = smelt_cuda_configure(ctx, &cfg);
            if (s) return s;
            ctx->pipelines.clear();
        }
    }

    auto shaped = [&](const char* base, int cols, bool typed) { return std::string(base) + (typed ? type : "") + ":" + std::to_string(cols) + ":" + std::to_string(W); };
    auto window = [&](Rec& r, const smelt_dense_layer& w, const LayerShape& s) {
        r.u32(8, (uint32_t)w.heads | ((uint32_t)w.kv_heads << 16)).u32(9, (uint32_t)w.dim | ((uint32_t)w.vdim << 16)).u32(10, w.window).u32(11, w.pool).u32(12, s.ring);
    };
    const uint8_t kSeq = SMELT_CONST_SEQ_LEN, kRows = SMELT_CONST_LOGIT_ROWS;
    {
        Rec r(e, "smelt_embed_positions", (W + 255) / 256, 1);
        r.buf(0, kWeights, d->embedding).buf(1, kTokenId).buf(2, kWeights, d->positions).buf(3, prefill ? (int)kDnPfX : SMELT_SLOT_CUR).buf(4, prefill ? kDnPfX0 : kDnEmbedding)
            .u32(5, W).u32(6, Wp).u32(8, d->max_positions).f32(9, d->embedding_scale);
        if (prefill) r.con(7, kSeq); else r.u32(7, 1);
    }
    for (size_t i = 0; i < runs.size(); ++i) {
        const smelt_dense_layer& w = layers[runs[i].layer];
        const LayerShape s = layer_shape(w, capacity, max_chunk);
        const int kslot = kKvBase + 2 * (int)i, vslot = kslot + 1, qv = w.heads * w.vdim, rows1 = s.qkv + w.ff;
        if (prefill) {
            const uint64_t z_ff = (uint64_t)qv * es;
            if (runs[i].begins) {
                Rec(e, "smelt_pair_rows" + type).buf(0, kDnPfX).buf(1, kDnPfX0).buf(2, kDnPfAct).u32(3, Wp).con(4, kSeq);
                Rec(e, shaped("smelt_dense_gemm", 2 * Wp, true)).buf(0, kWeights, d->loop_in).buf(1, kDnPfAct).buf(2, kDnPfX).u32(5, W).con(6, kSeq).u32(7, W).u32(8, Wp);
            }
            Rec(e, "smelt_scalar_norm_rows" + type).buf(0, kDnPfX).buf(1, kDnPfAct).u32(3, W).u32(4, Wp).con(5, kSeq).f32(6, w.norm_gain).f32(7, d->eps);
            Rec(e, shaped("smelt_dense_gemm_xielu", Wp, true)).buf(0, kWeights, w.in_proj).buf(1, kDnPfAct).buf(2, kDnPfU).buf(3, kDnPfZ, z_ff)
                .u32(5, rows1).con(6, kSeq).u32(7, s.qkv).u32(8, s.qkv).u32(9, s.cols2).f32(10, w.act_rising).f32(11, w.act_falling);
            { Rec r(e, "smelt_window_append" + type); r.buf(0, kDnPfU).buf(1, kWeights, w.q_norm).buf(2, kWeights, w.k_norm).buf(3, kslot).buf(4, vslot).buf(5, kDnPfQ); window(r, w, s); r.con(15, kSeq).f32(16, d->eps); }
            { Rec r(e, "smelt_window_pool" + type); r.buf(3, kslot).buf(4, vslot); window(r, w, s); r.con(15, kSeq); }
            { Rec r(e, shaped("smelt_window_attention", s.cols2, true)); r.buf(3, kslot).buf(4, vslot).buf(5, kDnPfQ).buf(6, kDnPfZ); window(r, w, s); r.f32(13, w.scale).f32(14, w.softcap).con(15, kSeq); }
            Rec(e, shaped("smelt_dense_gemm_add", s.cols2, true)).buf(0, kWeights, w.out_proj).buf(1, kDnPfZ).buf(2, kDnPfX).u32(5, W).con(6, kSeq).u32(7, W).u32(8, Wp);
        } else {
            if (runs[i].begins) {
                Rec(e, shaped("smelt_dense_matvec", 2 * Wp, false)).buf(0, kWeights, d->loop_in).buf(1, SMELT_SLOT_CUR).buf(2, kDnEmbedding).buf(3, SMELT_SLOT_ALT).u32(5, W);
                e.swap();
            }
            Rec(e, shaped("smelt_dense_matvec_xielu", Wp, false)).buf(0, kWeights, w.in_proj).buf(1, SMELT_SLOT_CUR).buf(3, kDnU).buf(4, kDnZ, (uint64_t)qv * 4)
                .u32(5, rows1).u32(6, s.qkv).f32(7, w.norm_gain).f32(8, d->eps).f32(9, w.act_rising).f32(10, w.act_falling);
            { Rec r(e, "smelt_window_decode" + type); r.buf(0, kDnU).buf(1, kWeights, w.q_norm).buf(2, kWeights, w.k_norm).buf(3, kslot).buf(4, vslot).buf(5, kDnQ).buf(6, kDnZ); window(r, w, s); r.f32(13, w.scale).f32(14, w.softcap).f32(16, d->eps); }
            Rec(e, shaped("smelt_dense_matvec_add", s.cols2, false)).buf(0, kWeights, w.out_proj).buf(1, kDnZ).buf(3, SMELT_SLOT_CUR).u32(5, W);
        }
    }
    if (prefill) {
        // the rows whose logits are asked for: final norm, head, argmax; skipped when there are none
        Rec(e, "smelt_scalar_norm_rows" + type).buf(0, kDnPfX).buf(1, kDnPfAct).buf(2, kLogitRowsSlot).u32(3, W).u32(4, Wp).con(5, kRows).f32(6, d->final_gain).f32(7, d->eps);
        Rec(e, shaped("smelt_dense_gemm", Wp, true)).buf(0, kWeights, d->lm_head).buf(1, kDnPfAct).buf(2, kLogits).u32(5, V).con(6, kRows).u32(7, V).u32(8, V);
        Rec(e, "argmax_f32_partials", parts).buf(0, kLogits).buf(1, kArgmaxScratch).u32(2, V).u32(3, chunk).con(4, kRows);
        Rec(e, "argmax_key_reduce", 1).buf(0, kArgmaxScratch).buf(1, kArgmax).u32(2, parts).con(4, kRows);
    } else {
        Rec(e, shaped("smelt_dense_matvec", Wp, false)).buf(0, kWeights, d->lm_head).buf(1, SMELT_SLOT_CUR).buf(3, kLogits).u32(5, V).f32(7, d->final_gain).f32(8, d->eps);
        Rec(e, "argmax_f32_partials", parts).buf(0, kLogits).buf(1, kArgmaxScratch).u32(2, V).u32(3, chunk).u32(4, 1);
        Rec(e, "argmax_key_reduce", 1).buf(0, kArgmaxScratch).buf(1, kArgmax).u32(2, parts);
    }
    const size_t need = e.n;
    if (records && need > *n_records) {
        *n_records = need;
        return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "build_dense: record buffer too small");
    }
    *n_records = need;
    if (names) {
        names->assign(e.pipes.size(), std::string());
        for (auto& kv : e.pipes) (*names)[kv.second - e.base] = kv.first;
    }
    return e.status;
}

}  // namespace

extern "C" smelt_status smelt_cuda_build_dense_decoder(smelt_cuda_ctx* ctx, const smelt_dense_desc* desc, const smelt_dense_layer* layers, uint32_t capacity,
                                                       uint32_t max_chunk, smelt_dispatch_record* records, size_t* n_records) {
    return build(ctx, desc, layers, capacity, max_chunk, false, records, n_records);
}

extern "C" smelt_status smelt_cuda_build_dense_prefill_table(smelt_cuda_ctx* ctx, const smelt_dense_desc* desc, const smelt_dense_layer* layers, uint32_t capacity,
                                                             uint32_t max_chunk, smelt_dispatch_record* records, size_t* n_records) {
    return build(ctx, desc, layers, capacity, max_chunk, true, records, n_records);
}

extern "C" smelt_status smelt_cuda_dense_cache_slots(const smelt_dense_desc* desc, int32_t* first_slot, int32_t* n_slots) {
    if (!desc || !first_slot || !n_slots || desc->loop_start < 0 || desc->loop_stop < desc->loop_start || desc->loop_stop > desc->layers || desc->loop_times < 0) return SMELT_ERR_BAD_ARGUMENT;
    *first_slot = kKvBase;
    *n_slots = 2 * (int32_t)layer_runs(desc).size();
    return SMELT_OK;
}

extern "C" smelt_status smelt_cuda_dense_slots(const smelt_dense_desc* desc, const smelt_dense_layer* layers, uint32_t capacity, uint32_t max_chunk, int32_t* slots,
                                               uint64_t* bytes, int32_t* n_slots) {
    if (!desc || !layers || !n_slots || validate(desc, layers, capacity, max_chunk)) return SMELT_ERR_BAD_ARGUMENT;
    std::map<int, size_t> all;
    for (bool prefill : {false, true})
        for (auto& p : slot_plan(desc, layers, capacity, max_chunk, prefill)) all[p.first] = std::max(all[p.first], p.second);
    const int32_t room = *n_slots;
    *n_slots = (int32_t)all.size();
    if (!slots || !bytes) return SMELT_OK;
    if (room < *n_slots) return SMELT_ERR_BAD_ARGUMENT;
    for (auto& p : all) { *slots++ = p.first; *bytes++ = p.second; }
    return SMELT_OK;
}

extern "C" smelt_status smelt_cuda_dense_pipelines(const smelt_dense_desc* desc, const smelt_dense_layer* layers, uint32_t capacity, uint32_t max_chunk, int prefill, char* out,
                                                   size_t out_bytes, size_t* needed_bytes) {
    if (!needed_bytes) return SMELT_ERR_BAD_ARGUMENT;
    std::vector<std::string> names;
    size_t n = 0;
    smelt_status s = build(nullptr, desc, layers, capacity, max_chunk, prefill != 0, nullptr, &n, &names);
    if (s) return s;
    std::string joined;
    for (auto& name : names) joined += name + "\n";
    *needed_bytes = joined.size() + 1;
    if (out && out_bytes >= joined.size() + 1) memcpy(out, joined.c_str(), joined.size() + 1);
    return SMELT_OK;
}
