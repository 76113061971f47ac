// Table builder for stacks of mixers and feed-forwards with dense 16-bit weights
// (smelt_cuda_build_stack_decoder): slots, pipelines and the decode and prompt-chunk records.
//
// Every sublayer's output is normed before it is added, so the sum belongs to the launch that reads
// the stream next: in a decode step to the next sublayer's first matrix-vector product (which swaps
// the two residual buffers), in a prompt chunk to the row kernel in front of it.
#include <algorithm>
#include <map>
#include <utility>
#include <vector>

#include "record_writer.h"
#include "stack.h"

using namespace smelt;

namespace {

enum StackSlot : int {
    kStU = 20, kStQ = 21, kStZ = 23, kStY = 24, kStH = 25, kStQa = 26, kStPart = 27, kStPartMl = 28, kStLogits = 18, kStChosen = 19,
    kStPfX = 2, kStPfY = 3, kStPfAct = 4, kStPfU = 5, kStPfQ = 6, kStPfZ = 7, kStPfH = 9, kStPfMix = 10, kStPfInner = 11, kStPfKv = 12, kStPfQa = 29, kStPfPart = 31,
    kStPfPartMl = 32, kStPfLogits = 37, kStPfChosen = 38, kStPfPlace = 39, kStPfTable = 14, kStPfPermuted = 15, kStPfRows = 13,
};

constexpr int kArgmaxChunk = 2048;

int pad128(int n) { return (n + 127) / 128 * 128; }

struct Shape {
    // latent
    int dp, rp, vp, kr, qp, in_rows;
    uint32_t ring;
    bool own, reads_others;
    // time mixing
    int hd, group, rank;
    // feed-forward
    int ffp;
    // output projection
    int cols2;
    int state = -1, state2 = -1;  // state slots
};

struct Plan {
    std::vector<Shape> layers;
    int n_state = 0;
};

Plan make_plan(const smelt_stack_desc* d, const smelt_stack_layer* layers, uint32_t max_chunk) {
    Plan p;
    std::vector<uint32_t> window(d->layers, 0);  // of every layer that reads a cache
    for (int l = 0; l < d->layers; ++l)
        if (layers[l].mixer == SMELT_MIXER_LATENT) {
            const int from = layers[l].kv_from >= 0 ? layers[l].kv_from : l;
            window[from] = std::max(window[from], layers[l].window);
        }
    for (int l = 0; l < d->layers; ++l) {
        const smelt_stack_layer& w = layers[l];
        Shape s = {};
        s.state = s.state2 = -1;
        if (w.mixer == SMELT_MIXER_LATENT) {
            s.dp = pad16(w.dim); s.rp = pad16(w.rot_dim); s.vp = latent_value_pad(w.vdim); s.kr = pad64(w.kv_rank); s.qp = pad64(w.q_rank);
            s.own = w.kv_from < 0;
            s.in_rows = s.qp + (s.own ? w.kv_rank + w.rot_dim : 0);
            s.cols2 = w.heads * s.vp;
            if (s.own) {
                s.ring = window_ring_rows(window[l], 1, max_chunk);
                s.state = kKvBase + p.n_state++;
                s.state2 = kKvBase + p.n_state++;
            } else {
                const Shape& f = p.layers[w.kv_from];
                s.ring = f.ring; s.state = f.state; s.state2 = f.state2;
            }
        } else {
            s.hd = w.heads * w.dim; s.group = pad128(s.hd); s.rank = pad64(w.rank);
            s.in_rows = 4 * s.group + s.rank;
            s.cols2 = pad64(s.hd);
            s.state = kKvBase + p.n_state++;
            s.state2 = kKvBase + p.n_state++;
        }
        s.ffp = w.ff_kind == SMELT_FF_NONE ? 0 : pad64(w.ff);
        p.layers.push_back(s);
    }
    return p;
}

const char* validate(const smelt_stack_desc* d, const smelt_stack_layer* layers, uint32_t capacity, uint32_t max_chunk) {
    if (d->layers <= 0 || d->width <= 0 || d->vocab <= 0 || capacity == 0 || capacity > 0x7FFFFFFFu || max_chunk == 0 || max_chunk > 1920) return "bad model size, capacity or chunk";
    if (d->precision != SMELT_DENSE_BF16 && d->precision != SMELT_DENSE_F32) return "unknown precision";
    for (int l = 0; l < d->layers; ++l) {
        const smelt_stack_layer& w = layers[l];
        if (w.heads <= 0 || w.dim <= 0 || w.heads > 65535 || w.dim > 65535) return "bad layer geometry";
        if (w.mixer == SMELT_MIXER_LATENT) {
            if (w.rot_dim <= 0 || w.rot_dims < 0 || w.rot_dims > w.rot_dim || w.rot_dims % 2 || w.vdim <= 0 || w.kv_rank <= 0 || w.q_rank <= 0 || w.window == 0 || w.rot_dim > 4096 ||
                w.vdim > 32768 || w.kv_rank > 32768 || w.q_rank > 32768 || w.window > 0x3FFFFFFFu)
                return "bad latent attention geometry";
            if (w.kv_from >= 0) {
                if (w.kv_from >= l) return "a layer reads the cache of a later one";
                const smelt_stack_layer& f = layers[w.kv_from];
                if (f.mixer != SMELT_MIXER_LATENT || f.kv_from >= 0 || f.kv_rank != w.kv_rank || f.rot_dim != w.rot_dim) return "a layer reads a cache that does not fit it";
            }
        } else if (w.mixer == SMELT_MIXER_WKV) {
            if (w.rank <= 0 || w.rank > 32768 || w.dim > 256) return "bad time mixing geometry";
        } else {
            return "unknown mixer";
        }
        if (w.ff_kind == SMELT_FF_NONE) continue;
        if (w.ff <= 0 || (w.ff_kind != SMELT_FF_DENSE && w.ff_kind != SMELT_FF_EXPERTS)) return "bad feed-forward";
        if (w.ff_kind == SMELT_FF_EXPERTS && (w.experts <= 0 || w.experts > 4096 || w.top <= 0 || w.top > w.experts || w.top > kMaxTop)) return "bad expert counts";
    }
    return nullptr;
}

using SlotPlan = std::vector<std::pair<int, size_t>>;

LatentArgs latent_shape(const smelt_stack_layer& w, const Shape& s, int m, bool decode) {
    LatentArgs a = {};
    a.heads = w.heads; a.kr = s.kr; a.rp = s.rp; a.window = w.window; a.m = m; a.q_f32 = decode; a.dp = s.dp; a.vp = s.vp;
    return a;
}
// The most key ranges a decode step of the layer may take on any GPU this is built for.
int max_splits(const smelt_stack_layer& w, const Shape& s, DenseType type) { return latent_splits(latent_shape(w, s, 1, true), type); }
bool tiled_prefill(const smelt_stack_layer& w, const Shape& s, DenseType type) { return type == kDenseBf16 && latent_prefill_tiled(latent_shape(w, s, 2, false)); }

// The slots one table binds, with their sizes.
SlotPlan slot_plan(const smelt_stack_desc* d, const smelt_stack_layer* layers, const Plan& p, uint32_t max_chunk, bool prefill) {
    const DenseType type = (DenseType)d->precision;
    const size_t Wp = pad64(d->width), V = d->vocab, es = type == kDenseF32 ? 4 : 2, parts = (V + kArgmaxChunk - 1) / kArgmaxChunk;
    std::map<int, size_t> sz;
    auto need = [&](int slot, size_t bytes) { sz[slot] = std::max(sz[slot], bytes); };
    if (prefill) {
        const size_t T = max_chunk;
        need(kStPfX, T * Wp * 4); need(kStPfY, T * Wp * 4); need(kStPfAct, T * Wp * es); need(kLogits, T * V * 4); need(kArgmaxScratch, T * parts * 8);
        need(kArgmax, std::max<size_t>(T * 4, 8)); need(kTokenId, T * 4); need(kLogitRowsSlot, T * 4);
        for (int l = 0; l < d->layers; ++l) {
            const smelt_stack_layer& w = layers[l];
            const Shape& s = p.layers[l];
            if (w.mixer == SMELT_MIXER_LATENT) {
                need(kStPfU, T * s.in_rows * 4);
                need(kStPfInner, T * s.qp * es);
                need(kStPfQ, T * w.heads * (s.dp + s.rp) * es);
                if (tiled_prefill(w, s, type)) {
                    need(kStPfKv, (size_t)s.ring * w.heads * (s.dp + s.vp) * es);
                } else {
                    need(kStPfQa, T * w.heads * (s.kr + s.rp) * 4);
                    need(kStPfPart, T * w.heads * s.kr * 4);
                    need(kStPfPartMl, T * w.heads * 8);
                }
            } else {
                need(kStPfU, T * 4 * s.group * 4);
                need(kStPfInner, T * s.rank * es);
                need(kStPfMix, 5 * T * Wp * es);
                need(kStPfH, T * Wp * 4);
                need(kStPfKv, T * s.hd * 4);  // decays
                need(kStPfPart, T * s.hd * 4);
            }
            need(kStPfZ, T * s.cols2 * es);
            if (w.ff_kind == SMELT_FF_DENSE) need(kStPfZ, T * s.ffp * es);
            if (w.ff_kind == SMELT_FF_EXPERTS) {
                const size_t pairs = T * w.top;
                need(kStPfLogits, T * w.experts * 4);
                need(kStPfChosen, pairs * 8);
                need(kStPfPlace, pairs * 4);
                need(kStPfTable, (1 + (size_t)w.experts + pairs) * 16);
                need(kStPfPermuted, pairs * Wp * es);
                need(kStPfZ, pairs * s.ffp * es);
                need(kStPfRows, pairs * Wp * 4);
            }
        }
    } else {
        need(kHiddenA, Wp * 4); need(kHiddenB, Wp * 4); need(kStY, Wp * 4); need(kLogits, V * 4); need(kArgmax, 8); need(kTokenId, 4); need(kPosition, 8); need(kArgmaxScratch, parts * 8);
        for (int l = 0; l < d->layers; ++l) {
            const smelt_stack_layer& w = layers[l];
            const Shape& s = p.layers[l];
            need(kStU, (size_t)s.in_rows * 4);
            need(kStZ, (size_t)std::max(s.cols2, w.ff_kind == SMELT_FF_EXPERTS ? w.top * s.ffp : s.ffp) * 4);
            if (w.mixer == SMELT_MIXER_LATENT) {
                const size_t splits = max_splits(w, s, type);
                need(kStQ, (size_t)w.heads * (s.dp + s.rp) * 4);
                need(kStQa, (size_t)w.heads * (s.kr + s.rp) * 4);
                need(kStPart, splits * w.heads * s.kr * 4);
                need(kStPartMl, splits * w.heads * 8);
                if (s.own) {
                    need(s.state, (size_t)s.ring * s.kr * es);
                    need(s.state2, (size_t)s.ring * s.rp * es);
                }
            } else {
                need(kStH, Wp * 4);
                need(s.state, (size_t)w.heads * w.dim * w.dim * 4);
                need(s.state2, Wp * 4);
            }
            if (w.ff_kind == SMELT_FF_EXPERTS) {
                need(kStH, Wp * 4);
                need(kStLogits, (size_t)w.experts * 4);
                need(kStChosen, (size_t)w.top * 8);
            }
        }
    }
    SlotPlan plan;
    for (auto& kv : sz) plan.push_back(kv);
    return plan;
}

smelt_status build(smelt_cuda_ctx* ctx, const smelt_stack_desc* d, const smelt_stack_layer* layers, uint32_t capacity, uint32_t max_chunk, bool prefill,
                   smelt_dispatch_record* records, size_t* n_records, std::vector<std::string>* names = nullptr) {
    if (!d || !layers || !n_records) return SMELT_ERR_BAD_ARGUMENT;
    if (const char* why = validate(d, layers, capacity, max_chunk)) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, std::string("build_stack: ") + why);
    const Plan p = make_plan(d, layers, max_chunk);
    const int W = d->width, Wp = pad64(W), V = d->vocab, chunk = kArgmaxChunk, parts = (V + chunk - 1) / chunk;
    const DenseType dtype = (DenseType)d->precision;
    const size_t es = dtype == kDenseF32 ? 4 : 2;
    const std::string type = dtype == kDenseF32 ? "_f32" : "_bf16";
    Emitter e{ctx, records, records ? *n_records : 0};
    if (ctx) {
        if (!records) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "build_stack: a context needs a record buffer (query the count with a null context)");
        if (cudaSetDevice(ctx->device) != cudaSuccess) return fail(ctx, SMELT_ERR_CUDA, "cudaSetDevice");
        if (!ctx->slots[kWeights].ptr) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "build_stack: upload the weights image to slot 30 first");
        if (kKvBase + p.n_state > (int)ctx->slots.size()) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "build_stack: too many layers for the slot table");
        if (prefill && (!ctx->configured || !ctx->slots[kStU].ptr)) return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "build_stack: build the decode table first");
        for (auto& s : slot_plan(d, layers, p, max_chunk, prefill)) {
            smelt_status st = smelt_cuda_alloc_slot(ctx, s.first, s.second);
            if (st) return st;
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

    auto shaped = [&](const char* base, int cols, int width, bool typed) { return std::string(base) + (typed ? type : "") + ":" + std::to_string(cols) + ":" + std::to_string(width); };
    const uint8_t kSeq = SMELT_CONST_SEQ_LEN, kRows = SMELT_CONST_LOGIT_ROWS;
    // geometry of a latent layer; q_rank travels as the name's second number
    auto latent = [&](Rec& r, const smelt_stack_layer& w, const Shape& s) {
        r.u32(20, (uint32_t)w.heads | (s.own ? 1u << 16 : 0u)).u32(21, (uint32_t)w.dim | ((uint32_t)w.rot_dim << 16)).u32(22, (uint32_t)w.vdim | ((uint32_t)w.rot_dims << 16))
            .u32(23, (uint32_t)w.kv_rank).u32(24, s.ring);
        if (prefill) r.con(25, kSeq); else r.u32(25, 1);
    };
    auto lname = [&](const char* base, const smelt_stack_layer& w, int cols) { return shaped(base, cols, w.q_rank, true); };
    auto wkv = [&](Rec& r, const smelt_stack_layer& w, const Shape& s) {
        r.u32(20, (uint32_t)w.heads | ((uint32_t)w.dim << 16)).u32(21, (uint32_t)s.rank).u32(22, (uint32_t)Wp);
        if (prefill) r.con(25, kSeq); else r.u32(25, 1);
    };

    // decode: the matrix-vector product that reads the stream, after the sublayer whose output is in kStY
    bool pending = false;  // kStY waits to be added, through this norm
    uint64_t pending_norm = 0;
    auto stream_matvec = [&](const char* base, uint64_t weights, uint64_t norm, int rows, int out_slot) {
        Rec r(e, shaped(base, Wp, W, false));
        r.buf(0, kWeights, weights).buf(1, SMELT_SLOT_CUR).buf(4, kWeights, norm).buf(8, out_slot).u32(10, (uint32_t)rows).f32(11, d->eps);
        if (pending) r.buf(2, kStY).buf(3, kWeights, pending_norm).buf(5, SMELT_SLOT_ALT);
        return r;
    };
    auto added = [&] { if (pending) e.swap(); pending = false; };
    auto plain_matvec = [&](uint64_t weights, int slot, int cols, int rows, uint64_t bias, bool has_bias, int out_slot) {
        Rec r(e, shaped("smelt_matvec", cols, cols, false));
        r.buf(0, kWeights, weights).buf(1, slot).buf(8, out_slot).u32(10, (uint32_t)rows);
        if (has_bias) r.buf(7, kWeights, bias);
    };
    // prompt chunk: the row kernel that adds kStPfY and norms
    auto row_norm = [&](uint64_t norm, bool h_f32, bool list) {
        Rec r(e, "smelt_residual_norm_rows" + type);
        r.buf(0, kStPfX).buf(3, kWeights, norm).buf(5, kStPfAct).u32(10, W).u32(11, Wp).f32(13, d->eps);
        if (pending) r.buf(1, kStPfY).buf(2, kWeights, pending_norm);
        if (list) r.buf(4, kLogitRowsSlot).con(12, kRows); else r.con(12, kSeq);
        if (h_f32) r.buf(6, kStPfH);
        pending = false;
    };
    auto gemm = [&](const char* base, uint64_t weights, int x_slot, int cols, int rows, int y_slot, int ld) {
        Rec r(e, shaped(base, cols, cols, true));
        r.buf(0, kWeights, weights).buf(1, x_slot).buf(2, y_slot).u32(5, (uint32_t)rows).u32(7, (uint32_t)rows).u32(8, (uint32_t)ld);
        return r;
    };

    {
        Rec r(e, "smelt_embed_rows", (W + 255) / 256, 1);
        r.buf(0, kWeights, d->embedding).buf(1, kTokenId).buf(2, prefill ? (int)kStPfX : SMELT_SLOT_CUR).u32(5, W).u32(6, Wp).f32(9, d->embedding_scale);
        if (prefill) r.con(7, kSeq); else r.u32(7, 1);
    }
    for (int l = 0; l < d->layers; ++l) {
        const smelt_stack_layer& w = layers[l];
        const Shape& s = p.layers[l];
        const uint64_t uv = w.kv_proj;
        if (!prefill) {
            if (w.mixer == SMELT_MIXER_LATENT) {
                stream_matvec("smelt_matvec_residual", w.in_proj, w.norm1, s.in_rows, kStU);
                added();
                Rec(e, shaped("smelt_matvec_norm", s.qp, w.q_rank, false)).buf(0, kWeights, w.q_proj).buf(1, kStU).buf(4, kWeights, w.q_norm).buf(8, kStQ)
                    .u32(10, (uint32_t)(w.heads * (s.dp + s.rp))).f32(11, d->eps);
                { Rec r(e, lname("smelt_latent_query", w, s.in_rows)); r.buf(0, kStU).buf(1, kStQ).buf(3, kWeights, uv).buf(4, s.state).buf(5, s.state2).buf(6, kStQa).buf(7, kWeights, w.rot_freq);
                  if (s.own) r.buf(2, kWeights, w.kv_norm); latent(r, w, s); r.f32(26, d->eps); }
                { Rec r(e, lname("smelt_latent_scores", w, s.in_rows)); r.buf(4, s.state).buf(5, s.state2).buf(6, kStQa).buf(8, kStPart).buf(9, kStPartMl); latent(r, w, s); r.u32(27, w.window).f32(28, w.scale); }
                { Rec r(e, lname("smelt_latent_values", w, s.cols2)); r.buf(3, kWeights, uv).buf(8, kStPart).buf(9, kStPartMl).buf(10, kStZ); latent(r, w, s); r.u32(27, w.window); }
            } else {
                { Rec r = stream_matvec("smelt_matvec_shift", w.in_proj, w.norm1, s.in_rows, kStU);
                  r.buf(6, kStH).buf(9, s.state2).buf(10, kWeights, w.mu).u32(12, (uint32_t)s.group); }
                added();
                { Rec r(e, "smelt_wkv_decode"); r.buf(0, kStU).buf(1, kWeights, w.w2).buf(2, kWeights, w.w0).buf(3, kWeights, w.bonus).buf(4, kWeights, w.head_norm).buf(5, s.state).buf(6, s.state2)
                      .buf(7, kStH).buf(8, kStZ); wkv(r, w, s); r.f32(26, d->eps); }
            }
            plain_matvec(w.out_proj, kStZ, s.cols2, W, 0, false, kStY);
            pending = true; pending_norm = w.norm1b;
            if (w.ff_kind == SMELT_FF_DENSE) {
                stream_matvec("smelt_matvec_residual", w.up, w.norm2, w.ff, kStZ).buf(7, kWeights, w.up_bias).u32(12, kActRelu2);
                added();
                plain_matvec(w.down, kStZ, s.ffp, W, w.down_bias, true, kStY);
            } else if (w.ff_kind == SMELT_FF_EXPERTS) {
                stream_matvec("smelt_matvec_residual", w.router, w.norm2, w.experts, kStLogits).buf(6, kStH).buf(7, kWeights, w.router_bias);
                added();
                Rec(e, shaped("smelt_matvec_experts_in", Wp, W, false)).buf(0, kWeights, w.up).buf(1, kStH).buf(6, kStLogits).buf(8, kStZ).buf(9, kStChosen)
                    .u32(10, (uint32_t)(2 * s.ffp)).u32(12, (uint32_t)w.experts).u32(13, (uint32_t)w.top).f32(14, w.limit);
                Rec(e, shaped("smelt_matvec_experts_out", s.ffp, w.ff, false)).buf(0, kWeights, w.down).buf(1, kStZ).buf(8, kStY).buf(9, kStChosen)
                    .u32(10, (uint32_t)W).u32(12, (uint32_t)w.experts).u32(13, (uint32_t)w.top);
            }
            if (w.ff_kind != SMELT_FF_NONE) { pending = true; pending_norm = w.norm2b; }
            continue;
        }
        row_norm(w.norm1, w.mixer == SMELT_MIXER_WKV, false);
        if (w.mixer == SMELT_MIXER_LATENT) {
            gemm("smelt_dense_gemm", w.in_proj, kStPfAct, Wp, s.in_rows, kStPfU, s.in_rows).con(6, kSeq);
            { Rec r(e, lname("smelt_latent_append", w, s.in_rows)); r.buf(0, kStPfU).buf(1, kWeights, w.q_norm).buf(4, s.state).buf(5, s.state2).buf(6, kStPfInner).buf(7, kWeights, w.rot_freq);
              if (s.own) r.buf(2, kWeights, w.kv_norm); latent(r, w, s); r.f32(26, d->eps); }
            const int q_rows = w.heads * (s.dp + s.rp);
            gemm("smelt_dense_gemm_act", w.q_proj, kStPfInner, s.qp, q_rows, kStPfQ, q_rows).con(6, kSeq);
            if (tiled_prefill(w, s, dtype)) {
                const int kv_rows = w.heads * (s.dp + s.vp);
                gemm("smelt_dense_gemm_ring", w.kv_proj, s.state, s.kr, kv_rows, kStPfKv, kv_rows).u32(6, s.ring);
                Rec r(e, lname("smelt_latent_prefill", w, s.cols2)); r.buf(1, kStPfQ).buf(5, s.state2).buf(7, kWeights, w.rot_freq).buf(8, kStPfKv).buf(10, kStPfZ); latent(r, w, s); r.u32(27, w.window).f32(28, w.scale);
            } else {
                { Rec r(e, lname("smelt_latent_query", w, s.in_rows)); r.buf(1, kStPfQ).buf(3, kWeights, uv).buf(4, s.state).buf(5, s.state2).buf(6, kStPfQa).buf(7, kWeights, w.rot_freq); latent(r, w, s); r.f32(26, d->eps); }
                { Rec r(e, lname("smelt_latent_scores", w, s.in_rows)); r.buf(4, s.state).buf(5, s.state2).buf(6, kStPfQa).buf(8, kStPfPart).buf(9, kStPfPartMl); latent(r, w, s); r.u32(27, w.window).f32(28, w.scale); }
                { Rec r(e, lname("smelt_latent_values", w, s.cols2)); r.buf(3, kWeights, uv).buf(8, kStPfPart).buf(9, kStPfPartMl).buf(10, kStPfZ); latent(r, w, s); r.u32(27, w.window); }
            }
        } else {
            { Rec r(e, "smelt_shift_mix_rows" + type); r.buf(6, s.state2).buf(7, kStPfH).buf(9, kWeights, w.mu).buf(10, kStPfMix); wkv(r, w, s); }
            Rec(e, shaped("smelt_dense_gemm_groups", Wp, s.group, true)).buf(0, kWeights, w.in_proj).buf(1, kStPfMix).buf(2, kStPfU).buf(3, kStPfInner).u32(5, (uint32_t)s.in_rows).con(6, kSeq)
                .u32(7, (uint32_t)(4 * s.group)).u32(8, (uint32_t)(4 * s.group)).u32(9, (uint32_t)s.rank).u32(12, kDenseTanh);
            gemm("smelt_dense_gemm_decay", w.w2, kStPfInner, s.rank, s.hd, kStPfKv, s.hd).con(6, kSeq).buf(4, kWeights, w.w0);
            { Rec r(e, "smelt_wkv_prefill"); r.buf(0, kStPfU).buf(3, kWeights, w.bonus).buf(5, s.state).buf(6, s.state2).buf(7, kStPfH).buf(8, kStPfPart).buf(11, kStPfKv); wkv(r, w, s); }
            { Rec r(e, "smelt_wkv_gate_rows" + type); r.buf(0, kStPfU).buf(4, kWeights, w.head_norm).buf(8, kStPfPart).buf(10, kStPfZ); wkv(r, w, s); r.f32(26, d->eps); }
        }
        gemm("smelt_dense_gemm", w.out_proj, kStPfZ, s.cols2, W, kStPfY, Wp).con(6, kSeq);
        pending = true; pending_norm = w.norm1b;
        if (w.ff_kind == SMELT_FF_DENSE) {
            row_norm(w.norm2, false, false);
            Rec(e, shaped("smelt_dense_gemm_relu2", Wp, W, true)).buf(0, kWeights, w.up).buf(1, kStPfAct).buf(2, kStPfZ).buf(3, kStPfZ).buf(4, kWeights, w.up_bias).u32(5, (uint32_t)w.ff).con(6, kSeq)
                .u32(7, 0).u32(8, (uint32_t)s.ffp).u32(9, (uint32_t)s.ffp).u32(12, kDenseRelu2);
            gemm("smelt_dense_gemm", w.down, kStPfZ, s.ffp, W, kStPfY, Wp).con(6, kSeq).buf(4, kWeights, w.down_bias);
        } else if (w.ff_kind == SMELT_FF_EXPERTS) {
            row_norm(w.norm2, false, false);
            gemm("smelt_dense_gemm", w.router, kStPfAct, Wp, w.experts, kStPfLogits, w.experts).con(6, kSeq).buf(4, kWeights, w.router_bias);
            auto moe = [&](const char* base, bool typed) {
                Rec r(e, shaped(base, Wp, W, typed));
                r.buf(4, kStPfChosen).buf(5, kStPfPlace).u32(10, (uint32_t)w.experts).u32(11, (uint32_t)w.top).con(12, kSeq);
                return r;
            };
            moe("smelt_moe_route", true).buf(3, kStPfLogits).buf(6, kStPfTable);
            moe("smelt_moe_gather", true).buf(1, kStPfAct).buf(2, kStPfPermuted);
            auto expert_gemm = [&](const char* base, int cols, int rows, uint64_t weights, int x, int y, int ld) {
                Rec r(e, shaped(base, cols, cols, true));
                r.buf(0, kWeights, weights).buf(1, x).buf(2, y).buf(6, kStPfTable).u32(5, (uint32_t)rows).con(6, kSeq).u32(8, (uint32_t)ld).u32(10, (uint32_t)w.experts).u32(11, (uint32_t)w.top);
                return r;
            };
            expert_gemm("smelt_expert_gemm_glu", Wp, 2 * s.ffp, w.up, kStPfPermuted, kStPfZ, s.ffp).f32(13, w.limit);
            expert_gemm("smelt_expert_gemm", s.ffp, W, w.down, kStPfZ, kStPfRows, Wp);
            moe("smelt_moe_combine", false).buf(7, kStPfRows).buf(8, kStPfY);
        }
        if (w.ff_kind != SMELT_FF_NONE) { pending = true; pending_norm = w.norm2b; }
    }
    if (prefill) {
        // the rows whose logits are asked for: residual, final norm, head, argmax; skipped when there are none
        row_norm(d->final_norm, false, true);
        gemm("smelt_dense_gemm", d->lm_head, kStPfAct, Wp, V, kLogits, V).con(6, kRows);
        Rec(e, "argmax_f32_partials", parts).buf(0, kLogits).buf(1, kArgmaxScratch).u32(2, V).u32(3, chunk).con(4, kRows);
        Rec(e, "argmax_key_reduce", 1).buf(0, kArgmaxScratch).buf(1, kArgmax).u32(2, parts).con(4, kRows);
    } else {
        stream_matvec("smelt_matvec_residual", d->lm_head, d->final_norm, V, kLogits);
        Rec(e, "argmax_f32_partials", parts).buf(0, kLogits).buf(1, kArgmaxScratch).u32(2, V).u32(3, chunk).u32(4, 1);
        Rec(e, "argmax_key_reduce", 1).buf(0, kArgmaxScratch).buf(1, kArgmax).u32(2, parts);
    }
    const size_t need = e.n;
    if (records && need > *n_records) {
        *n_records = need;
        return fail(ctx, SMELT_ERR_BAD_ARGUMENT, "build_stack: record buffer too small");
    }
    *n_records = need;
    if (names) {
        names->assign(e.pipes.size(), std::string());
        for (auto& kv : e.pipes) (*names)[kv.second - e.base] = kv.first;
    }
    (void)es;
    return e.status;
}

}  // namespace

extern "C" smelt_status smelt_cuda_build_stack_decoder(smelt_cuda_ctx* ctx, const smelt_stack_desc* desc, const smelt_stack_layer* layers, uint32_t capacity,
                                                       uint32_t max_chunk, smelt_dispatch_record* records, size_t* n_records) {
    return build(ctx, desc, layers, capacity, max_chunk, false, records, n_records);
}

extern "C" smelt_status smelt_cuda_build_stack_prefill_table(smelt_cuda_ctx* ctx, const smelt_stack_desc* desc, const smelt_stack_layer* layers, uint32_t capacity,
                                                             uint32_t max_chunk, smelt_dispatch_record* records, size_t* n_records) {
    return build(ctx, desc, layers, capacity, max_chunk, true, records, n_records);
}

extern "C" smelt_status smelt_cuda_stack_cache_slots(const smelt_stack_desc* desc, const smelt_stack_layer* layers, int32_t* first_slot, int32_t* n_slots) {
    if (!desc || !layers || !first_slot || !n_slots || validate(desc, layers, 1, 1)) return SMELT_ERR_BAD_ARGUMENT;
    *first_slot = kKvBase;
    *n_slots = make_plan(desc, layers, 1).n_state;
    return SMELT_OK;
}

extern "C" smelt_status smelt_cuda_stack_slots(const smelt_stack_desc* desc, const smelt_stack_layer* layers, uint32_t capacity, uint32_t max_chunk, int32_t* slots,
                                               uint64_t* bytes, int32_t* n_slots) {
    if (!desc || !layers || !n_slots || validate(desc, layers, capacity, max_chunk)) return SMELT_ERR_BAD_ARGUMENT;
    const Plan p = make_plan(desc, layers, max_chunk);
    std::map<int, size_t> all;
    for (bool prefill : {false, true})
        for (auto& s : slot_plan(desc, layers, p, max_chunk, prefill)) all[s.first] = std::max(all[s.first], s.second);
    const int32_t room = *n_slots;
    *n_slots = (int32_t)all.size();
    if (!slots || !bytes) return SMELT_OK;
    if (room < *n_slots) return SMELT_ERR_BAD_ARGUMENT;
    for (auto& s : all) { *slots++ = s.first; *bytes++ = s.second; }
    return SMELT_OK;
}

extern "C" smelt_status smelt_cuda_stack_pipelines(const smelt_stack_desc* desc, const smelt_stack_layer* layers, uint32_t capacity, uint32_t max_chunk, int prefill, char* out,
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
