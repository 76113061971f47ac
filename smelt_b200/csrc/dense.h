// Decoders with dense 16-bit weights: bf16 matrices, fp32 residual stream, and either bf16 or
// fp32 activations and caches.  Launchers of dense_matvec.cu, dense_gemm.cu, dense_glue.cu and
// window_attention.cu.
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"

namespace smelt {

using bf16 = __nv_bfloat16;

// Element type of the activations and caches of one table.
enum DenseType : int { kDenseBf16 = 0, kDenseF32 = 1 };

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <class T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float exp2_approx(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// xIELU: rising * z^2 + z / 2 for z > 0, falling * (exp(z) - 1 - z) + z / 2 otherwise, where
// rising = softplus(p) and falling = 1 / 2 + softplus(q) of the layer's two stored numbers.
__device__ __forceinline__ float xielu(float z, float rising, float falling) {
    const float curve = z > 0.f ? rising * z * z : falling * (expm1f(z) - z);
    return fmaf(0.5f, z, curve);
}

// Where a projection's output rows go.  Rows below `split` to y0 (row-major [M, ld0]); rows from
// `split` on through an activation to y1 ([M, ld1]).  split == rows when there is no second part.
enum DenseMode : int {
    kDenseStoreF32 = 0,    // y0 fp32
    kDenseAddF32 = 1,      // y0 fp32, added to
    kDenseStoreAct = 2,    // y0 and y1 in the activations' type
    kDenseStoreMixed = 3,  // y0 fp32, y1 in the activations' type
    kDenseStoreGlu = 4,    // rows are (gate, up) pairs: y0[row / 2] = clamped_glu, in the activations' type
};
// Applied to the rows from `split` on; in kDenseStoreF32 kDenseDecay applies to all rows.
enum DenseAct : int { kDenseXielu = 0, kDenseRelu2 = 1, kDenseTanh = 2, kDenseDecay = 3 };
struct DenseOut {
    void* y0;
    void* y1;
    int ld0, ld1, split;
    float rising, falling;  // xIELU; kDenseStoreGlu: rising is the clamp's limit
    int act;
    const bf16* bias;       // per row, added first; null: none (kDenseAddF32 takes none)
};

// The clamped gate of a pair: g = min(g, limit), u = clamp(u, -limit, limit), g sigmoid(1.702 g) (u + 1).
__device__ __forceinline__ float clamped_glu(float g, float u, float limit) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.f + expf(-1.702f * g)) * (u + 1.f);
}

// y[rows] = W[rows, cols] . x, one activation row, everything but the weights in fp32 (both
// activation types use it: a decode step keeps its activations in fp32).  cols is a multiple of
// 64, x zero-padded up to it.  xb != null: x is [xa (ka values); xb (cols - ka)].  norm: the row
// is scaled by gain / rms(x), the mean taken over `width` values.
struct DenseMatvecArgs {
    const bf16* w;
    const float* xa;
    const float* xb;
    int ka;
    int rows, cols;
    int norm, width;
    float gain, eps;
    DenseOut out;
    int sm_count;
    DevDyn dyn;
};
cudaError_t launch_dense_matvec(const Launch& l, int mode, DenseMatvecArgs a);

// Y[m, rows] = X[m, cols] . W[rows, cols]^T for the m activation rows of a prompt chunk.  X in
// the activations' type with leading dimension cols (a multiple of 64, zero-padded).
struct DenseGemmArgs {
    const bf16* w;
    const void* x;
    int rows, cols, m;
    DenseOut out;
    int sm_count;
    uint32_t* err;
    float* part_scratch;       // split-K partial sums and arrival counters
    size_t part_scratch_bytes;
    int* part_counters;
    // Groups of rows with activations of their own: rows [g group_rows, (g + 1) group_rows) read X from row g x_group on, the last
    // of the `groups` has the rest of the rows (group_rows a multiple of 128; 0: one X).
    int group_rows, x_group, groups;
    // Experts: `rows` are one expert's, W holds `experts` of them one behind the other; table[0].x entries follow, each
    // {expert, first row of X and of y, rows (at most tile), 0}.  m: all rows of X.
    const int4* table;
    int experts, tile, max_entries;
};
cudaError_t launch_dense_gemm(const Launch& l, DenseType type, int mode, const DenseGemmArgs& a);

// x[r] = x0[r] = table[token[r]] * scale + pos_table[position + r]; rows of ld floats, width used.
cudaError_t launch_embed_positions(const Launch& l, const bf16* table, const int32_t* tokens, const bf16* pos_table, float* x, float* x0, int width, int ld, int m, uint32_t vocab, uint32_t max_positions, float scale);
// out[r] = x[rows ? rows[r] : r] * gain / rms, in the activations' type.
cudaError_t launch_scalar_norm_rows(const Launch& l, DenseType type, const float* x, const int32_t* rows, void* out, int width, int ld, int m, float gain, float eps);
// out[r] = [x[r]; x0[r]], 2 ld values.
cudaError_t launch_pair_rows(const Launch& l, DenseType type, const float* x, const float* x0, void* out, int ld, int m);
cudaError_t launch_argmax_f32_partials(const Launch& l, const float* logits, uint64_t* partials, int vocab, int chunk, int rows);

// Attention over a sliding window and pooled blocks.
//
// Cache of one layer run, per KV head: `ring` rows of tokens (position p in row p % ring), then
// `blocks` rows of block means (block b, the positions [b pool, b pool + pool), in row ring + b).
// Rows are kp / vp elements long, zero beyond dim / vdim.  A query at position i sees positions
// j with 0 <= i - j < window and blocks with b pool + pool - 1 <= i - window.
struct WindowArgs {
    int heads, kv_heads, dim, vdim, kp, vp;
    uint32_t window, pool, ring, blocks;
    float scale, softcap, eps;  // softcap <= 0: none
    int m;                      // query rows: positions dyn position .. + m - 1
    const void* u;              // [m, heads dim + kv_heads (dim + vdim)]: q | k | v projections
    int u_f32;                  // u, q and z in fp32 whatever the cache holds (a decode step)
    const bf16* q_norm;
    const bf16* k_norm;
    void* k_cache;
    void* v_cache;
    void* q;                    // [m, heads, kp] normed queries
    void* z;                    // [m, ldz]: the heads' outputs in columns [0, heads vdim)
    int ldz;
    int sm_count;
    DevDyn dyn;
};
inline int window_padded(int d) { return d <= 64 ? 64 : d <= 128 ? 128 : d <= 256 ? 256 : (d + 63) / 64 * 64; }
// Ring rows that a chunk of up to max_chunk positions needs.
inline uint32_t window_ring_rows(uint32_t window, uint32_t pool, uint32_t max_chunk) {
    const uint32_t keep = window > pool ? window : pool;
    return (keep + max_chunk + 63u) / 64u * 64u;
}
// Query and key norm per head; queries to q, keys and values into the ring.
cudaError_t launch_window_append(const Launch& l, DenseType type, WindowArgs a);
// Means of the blocks that the rows just appended complete.
cudaError_t launch_window_pool(const Launch& l, DenseType type, WindowArgs a);
cudaError_t launch_window_attention(const Launch& l, DenseType type, WindowArgs a);
// One decode step: norms, append, block mean and attention.
cudaError_t launch_window_decode(const Launch& l, DenseType type, WindowArgs a, int* launches);

template <class Kernel, class... Args>
inline cudaError_t launch_chained(const Launch& l, Kernel kernel, dim3 grid, dim3 block, size_t smem, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = l.stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = l.pdl ? 1 : 0;
    if (smem > 16 * 1024) {  // the default limit is 48 KB together with the kernel's static shared memory
        cudaError_t e = cudaFuncSetAttribute(reinterpret_cast<const void*>(kernel), cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
    }
    prefer_max_shared(kernel);
    return cudaLaunchKernelEx(&cfg, kernel, args...);
}

}  // namespace smelt
