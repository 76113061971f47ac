// Decoders whose layers are a mixer and a feed-forward in turn, each between a norm before and a
// norm after it: latent (MLA-style) window attention, RWKV-style time mixing, squared-ReLU and
// mixture-of-experts feed-forwards.  Launchers of stack_matvec.cu, stack_glue.cu, latent_*.cu, wkv.cu
// and moe.cu; the projections of a prompt chunk are dense_gemm.cu's.
#pragma once
#include "dense.h"

namespace smelt {

// ── decode: matrix-vector products with what surrounds them ─────────────────
// What the activation row is made of.
enum StackInput : int {
    kInPlain = 0,     // x
    kInNorm = 1,      // unit rms of x times norm_w
    kInResidual = 2,  // s = x + rms-norm(y) (1 + post_w), to x_out; h = rms-norm(s) (1 + norm_w), to h_out (y null: s = x, not written)
    kInShift = 3,     // the same, then per group of rows h + (before - h) mu[group]; before counts as zero at position 0
    kInExpertsIn = 4, // x; rows [gate; up] pairs of the chosen experts, top-k from `logits`
    kInExpertsOut = 5 // x = [top][cols of one expert]; the chosen experts' columns
};
enum StackAct : int { kActNone = 0, kActRelu2 = 1, kActGlu = 2 };

struct StackMatvecArgs {
    const bf16* w;
    int rows, cols, width;  // cols: a multiple of 64; kInExperts*: rows and cols of one expert
    const float* x;
    const float* y;
    const bf16* post_w;
    const bf16* norm_w;
    float* x_out;
    float* h_out;
    float eps;
    const float* before;
    const bf16* mu;      // [kMixes][cols]
    int group_rows;      // rows of each group but the last
    const bf16* bias;    // per row, or null
    int act;
    float* out;
    const float* logits; // [experts]
    int experts, top;
    float limit;
    int2* chosen;        // [top]: expert, weight bits; written by kInExpertsIn, read by kInExpertsOut
    int sm_count;
    DevDyn dyn;
};
constexpr int kMaxTop = 64;
constexpr int kMixes = 5;  // r, k, v, g, decay: groups of rows of the time mixing's input projection
cudaError_t launch_stack_matvec(const Launch& l, int input, StackMatvecArgs a);

__device__ __forceinline__ float silu(float z) { return z / (1.f + expf(-z)); }

// ── prompt chunks: row kernels ──────────────────────────────────────────────
// x[r] = table[token[r]] * scale.
cudaError_t launch_embed_rows(const Launch& l, const bf16* table, const int32_t* tokens, float* x, int width, int ld, int m, uint32_t vocab, float scale);
// s = x + rms-norm(y) (1 + post_w) (y null: s = x); h = rms-norm(s) (1 + norm_w), to out (activations' type) and to h_f32 (if not null).
// rows != null: only those rows, x is left as it is; otherwise x = s.
struct ResidualNormArgs {
    float* x;
    const float* y;
    const bf16* post_w;
    const bf16* norm_w;
    const int32_t* rows;
    void* out;
    float* h_f32;
    int width, ld, m;
    float eps;
    DevDyn dyn;
};
cudaError_t launch_residual_norm_rows(const Launch& l, DenseType type, ResidualNormArgs a);

// ── latent attention ────────────────────────────────────────────────────────
// Per head `dim` plain and `rot` rotated query elements, in rows of dp + rp (each a multiple of 16,
// zero padded); values vp wide (64, 128, 256 or a multiple of 64).  Cache: `ring` rows of latents
// (kr = rank padded to 64 elements) and of rotated key parts (rp elements); position p in row p % ring.
// freq: rot_dims / 2 doubles, the angle of pair i at position p is p freq[i].
struct LatentArgs {
    int heads, dim, rot, rot_dims, vdim, rank, q_rank, dp, rp, vp, kr, qp;  // qp: q_rank padded to 64
    uint32_t window, ring;
    float scale, eps;
    int m, own;         // own: u carries this layer's own latent and key part
    const float* u;     // [m, ldu]: query latent (qp) | latent (rank) | key part (rot)
    int ldu;
    const bf16* q_norm;
    const bf16* kv_norm;
    const double* freq;
    void* cq;           // [m, qp] normed query latents, activations' type
    const void* q;      // [m, heads (dp + rp)]: fp32 in a decode step, else the activations' type
    int q_f32;
    const bf16* kv;     // [uk: heads dp; uv: heads vp] x kr
    void* c_ring;
    void* rot_ring;
    float* qa;          // [m, heads, kr + rp] queries against the latents, rotated parts behind
    float* part;        // [m, splits, heads, kr] sums over the splits' keys
    float2* part_ml;    // [m, splits, heads]: running maximum and weight sum
    int splits;
    const void* kv_rows;  // [ring rows, heads (dp + vp)] keys and values of the latents (tiled prompt kernel)
    void* z;            // [m, ldz] the heads' outputs, vp columns each
    int ldz;
    int sm_count;
    DevDyn dyn;
};
inline int pad16(int n) { return (n + 15) / 16 * 16; }
inline int pad64(int n) { return (n + 63) / 64 * 64; }
inline int latent_value_pad(int vdim) { return window_padded(vdim); }
// The tensor-core kernels take these shapes.
inline bool latent_decode_tiled(const LatentArgs& a) { return a.kr <= 512 && a.rp <= 128; }
inline bool latent_prefill_tiled(const LatentArgs& a) { return a.dp + a.rp <= 320 && a.vp <= 256; }
// Key ranges of a decode step, from the geometry alone.
int latent_splits(const LatentArgs& a, DenseType type);
constexpr int kLatentTile = 32;  // keys of a decode tile
// Normed query latents, and (own) latents and rotated key parts into the ring.
cudaError_t launch_latent_append(const Launch& l, DenseType type, LatentArgs a);
// qa = each head's query through uk, its rotated part rotated.  append: a decode step, which also appends u's row.
cudaError_t launch_latent_query(const Launch& l, DenseType type, LatentArgs a, bool append);
// part = attention over the latents.
cudaError_t launch_latent_scores(const Launch& l, DenseType type, LatentArgs a);
// z = the splits of part merged, through uv.
cudaError_t launch_latent_values(const Launch& l, DenseType type, LatentArgs a);
// The prompt chunk's attention over kv_rows and rot_ring on the tensor cores (bf16).
cudaError_t launch_latent_prefill(const Launch& l, LatentArgs a);
cudaError_t launch_latent_decode_tiled(const Launch& l, const LatentArgs& a);

// ── time mixing ─────────────────────────────────────────────────────────────
// u: [m, ldu] projections, groups of `group` rows r | k | v | g, then the decay's inner values.
struct WkvArgs {
    int heads, dim, group, ldu, rank, ld, m;  // rank: padded to 64; ld: of h and before
    const float* u;
    const bf16* w2;      // [heads dim, rank]
    const bf16* w0;
    const bf16* bonus;
    const bf16* norm;
    const float* decay;  // [m, heads dim] decays (prompt chunks)
    float* state;        // [heads][key][value]
    float* before;       // [ld]: the previous token's h, written from the last row of h
    const float* h;
    const bf16* mu;      // [5][ld]
    void* out;           // decode: z fp32; shift: [5][m][ld] mixes; prefill: o fp32; gate: z in the activations' type
    const float* o;
    int ldz;
    float eps;
    int sm_count;
    DevDyn dyn;
};
cudaError_t launch_wkv_decode(const Launch& l, WkvArgs a);
cudaError_t launch_shift_mix_rows(const Launch& l, DenseType type, WkvArgs a);
cudaError_t launch_wkv_prefill(const Launch& l, WkvArgs a);
cudaError_t launch_wkv_gate_rows(const Launch& l, DenseType type, WkvArgs a);

// ── mixture of experts of a prompt chunk ────────────────────────────────────
// Every (token, chosen expert) pair gets a row of a permuted chunk in which an expert's rows are neighbours.
struct MoeArgs {
    int m, experts, top, tile;  // tile: rows of a table entry
    const float* logits;        // [m, experts]
    int2* chosen;               // [m, top]: expert, weight bits
    int32_t* place;             // [m, top]: permuted row
    int4* table;                // [0].x = entries; then {expert, first row, rows, 0}
    const void* h;              // [m, ld] activations
    void* permuted;             // [m top, ld]
    const float* y_rows;        // [m top, ld]
    float* y;                   // [m, ld]
    int width, ld;
    DevDyn dyn;
};
inline int moe_tile(int m, int top, int experts, DenseType type) {
    const long per = ((long)m * top + experts - 1) / experts;
    return type == kDenseF32 ? 64 : per <= 32 ? 32 : per <= 96 ? 64 : 128;
}
inline int moe_max_entries(int m, int top, int experts, int tile) { return experts + (int)(((long)m * top + tile - 1) / tile); }
cudaError_t launch_moe_route(const Launch& l, MoeArgs a);
cudaError_t launch_moe_gather(const Launch& l, DenseType type, MoeArgs a);
cudaError_t launch_moe_combine(const Launch& l, MoeArgs a);

}  // namespace smelt
