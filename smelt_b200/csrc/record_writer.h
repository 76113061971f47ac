// Writes SmeltDispatchRecord sequences: pipeline registration in order of first use, records with
// their buffer and constant bindings, and the slot numbers the decoder tables share
// (SmeltFixedSlot, Sources/SmeltCompiler/SmeltBufferPlan.swift:129-198).
#pragma once

#include <cstring>
#include <map>
#include <string>

#include "runtime.h"

namespace smelt {

enum FixedSlot : int {
    kHiddenA = 0, kHiddenB = 1, kNormOut = 8, kFfnInt = 13, kFfnDown = 14, kLogits = 16, kArgmax = 17,
    kAttnQ = 20, kAttnK = 21, kAttnV = 22, kAttnOut = 23, kWeights = 30,
    kTokenId = 33, kPosition = 34, kArgmaxScratch = 35, kKvBase = 40,
};

inline uint32_t f32_bits(float f) { uint32_t u; memcpy(&u, &f, 4); return u; }

struct Emitter {
    smelt_cuda_ctx* ctx;
    smelt_dispatch_record* out;
    size_t cap, n = 0;
    std::map<std::string, int> pipes;
    smelt_status status = SMELT_OK;
    int base = 0;  // first pipeline index this table may register (a prefill table comes after the decode table's)

    int pipe(const std::string& name) {
        auto it = pipes.find(name);
        if (it != pipes.end()) return it->second;
        const int idx = base + (int)pipes.size();
        if (ctx) {
            smelt_status s = smelt_cuda_register_pipeline(ctx, idx, name.c_str());
            if (s && !status) status = s;
        }
        pipes[name] = idx;
        return idx;
    }
    smelt_dispatch_record* next() {
        static smelt_dispatch_record scratch;
        smelt_dispatch_record* r = (out && n < cap) ? &out[n] : &scratch;
        memset(r, 0, sizeof(*r));
        ++n;
        return r;
    }
    void swap() { next()->op_kind = SMELT_OP_SWAP; }
};

struct Rec {
    smelt_dispatch_record* r;
    Rec(Emitter& e, const std::string& name, uint32_t gx = 1, uint32_t gy = 1) : r(e.next()) {
        r->op_kind = SMELT_OP_DISPATCH;
        r->pipeline = (uint16_t)e.pipe(name);
        r->grid[0] = gx; r->grid[1] = gy; r->grid[2] = 1;
        r->threadgroup[0] = 64; r->threadgroup[1] = 1; r->threadgroup[2] = 1;
    }
    Rec& buf(int binding, int slot, uint64_t offset = 0) {
        smelt_buffer_record& b = r->buf[r->buffer_count++];
        b.slot = (int16_t)slot; b.binding_index = (uint8_t)binding; b.offset_kind = 0; b.offset = offset;
        return *this;
    }
    Rec& con(int binding, uint8_t kind, uint32_t value = 0) {
        smelt_constant_record& c = r->con[r->constant_count++];
        c.kind = kind; c.binding_index = (uint8_t)binding; c.value = value;
        return *this;
    }
    Rec& u32(int binding, uint32_t v) { return con(binding, SMELT_CONST_LITERAL_U32, v); }
    // grid dimension `dim` follows the chunk length: kind 1 seqLen, 2 seqLen * literal, 3 ceil(seqLen / literal) (SmeltDispatchTable.swift:163-222)
    Rec& grid_kind(int dim, uint8_t kind) { r->style = (uint8_t)(r->style | (kind << (2 + 2 * dim))); return *this; }
    Rec& buf_kind(int binding, int slot, uint8_t kind, uint64_t offset) {
        buf(binding, slot, offset);
        r->buf[r->buffer_count - 1].offset_kind = kind;
        return *this;
    }
    Rec& tg(uint32_t w) { r->threadgroup[0] = w; return *this; }
    Rec& f32(int binding, float v) { return con(binding, SMELT_CONST_LITERAL_F32, f32_bits(v)); }
    Rec& affine(int first, const smelt_affine_ref& w) {
        return buf(first, kWeights, w.packed).buf(first + 1, kWeights, w.scales).buf(first + 2, kWeights, w.biases);
    }
};

}  // namespace smelt
