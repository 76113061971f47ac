// Row kernels of the dense-weight decoders: embedding with learned positions, the one-number RMS
// norm, the pair [x; x0] that enters a loop pass, and the argmax of fp32 logits.
#include "dense.h"

namespace smelt {

namespace {

constexpr int kRowThreads = 256;

__global__ void __launch_bounds__(kRowThreads) embed_positions_kernel(const bf16* table, const int32_t* tokens, const bf16* pos_table, float* x, float* x0,
                                                                      int width, int ld, uint32_t vocab, uint32_t max_positions, float scale, DevDyn dyn) {
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(dyn)) return;
    const uint32_t r = blockIdx.y, tok = (uint32_t)tokens[r], pos = dyn_position(dyn) + r;
    const int i = blockIdx.x * kRowThreads + threadIdx.x;
    if (i >= width || tok >= vocab || pos >= max_positions) return;  // the host validates both
    const float v = fmaf(to_f32(table[(size_t)tok * width + i]), scale, to_f32(pos_table[(size_t)pos * width + i]));
    x[(size_t)r * ld + i] = v;
    x0[(size_t)r * ld + i] = v;
}

// One warp per row.
template <class T>
__global__ void __launch_bounds__(kRowThreads) scalar_norm_rows_kernel(const float* __restrict__ x, const int32_t* rows, T* __restrict__ out, int width, int ld,
                                                                       int m, float gain, float eps, DevDyn dyn) {
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(dyn)) return;
    const int r = blockIdx.x * (kRowThreads / 32) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (r >= m) return;
    const float4* src = reinterpret_cast<const float4*>(x + (size_t)(rows ? rows[r] : r) * ld);
    float ss = 0.f;
    for (int i = lane; i < ld / 4; i += 32) {
        const float4 v = src[i];
        ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    }
    const float f = gain * rsqrtf(warp_sum(ss) / (float)width + eps);
    T* dst = out + (size_t)r * ld;
    for (int i = lane; i < ld / 4; i += 32) {
        const float4 v = src[i];
        if constexpr (sizeof(T) == 4) {
            reinterpret_cast<float4*>(dst)[i] = make_float4(v.x * f, v.y * f, v.z * f, v.w * f);
        } else {
            const __nv_bfloat162 a = __floats2bfloat162_rn(v.x * f, v.y * f), b = __floats2bfloat162_rn(v.z * f, v.w * f);
            reinterpret_cast<uint2*>(dst)[i] = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
        }
    }
}

template <class T>
__global__ void __launch_bounds__(kRowThreads) pair_rows_kernel(const float* __restrict__ x, const float* __restrict__ x0, T* __restrict__ out, int ld, DevDyn dyn) {
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(dyn)) return;
    const int i = blockIdx.x * kRowThreads + threadIdx.x;
    const size_t r = blockIdx.y;
    if (i >= 2 * ld) return;
    out[r * 2 * ld + i] = from_f32<T>(i < ld ? x[r * ld + i] : x0[r * ld + (i - ld)]);
}

// Orders a logit and its index: the larger value wins, ties go to the lower index, -0 equals +0.
__device__ __forceinline__ uint64_t argmax_key_f32(float v, uint32_t index) {
    uint32_t bits = __float_as_uint(v);
    if ((bits & 0x7FFFFFFFu) == 0u) bits = 0u;
    const uint32_t ordered = (bits & 0x80000000u) ? ~bits : (bits | 0x80000000u);
    return ((uint64_t)ordered << 32) | (uint64_t)(0xFFFFFFFFu - index);
}

__global__ void __launch_bounds__(kRowThreads) argmax_f32_partials_kernel(const float* __restrict__ logits, uint64_t* __restrict__ partials, int vocab, int chunk, DevDyn dyn) {
    __shared__ uint64_t sbest[kRowThreads / 32];
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(dyn)) return;
    const float* lg = logits + (size_t)blockIdx.y * vocab;
    const int start = blockIdx.x * chunk, end = min(start + chunk, vocab);
    uint64_t best = 0;
    for (int i = start + threadIdx.x; i < end; i += kRowThreads) {
        const uint64_t k = argmax_key_f32(lg[i], (uint32_t)i);
        best = k > best ? k : best;
    }
    for (int o = 16; o > 0; o >>= 1) {
        const uint64_t other = __shfl_xor_sync(0xffffffffu, best, o);
        best = other > best ? other : best;
    }
    if ((threadIdx.x & 31) == 0) sbest[threadIdx.x >> 5] = best;
    __syncthreads();
    if (threadIdx.x == 0) {
        for (int w = 1; w < kRowThreads / 32; ++w) best = sbest[w] > best ? sbest[w] : best;
        partials[(size_t)blockIdx.y * gridDim.x + blockIdx.x] = best;
    }
}

}  // namespace

cudaError_t launch_embed_positions(const Launch& l, const bf16* table, const int32_t* tokens, const bf16* pos_table, float* x, float* x0, int width, int ld, int m,
                                   uint32_t vocab, uint32_t max_positions, float scale) {
    if (width <= 0 || ld < width || m <= 0) return cudaErrorInvalidValue;
    return launch_chained(l, embed_positions_kernel, dim3((width + kRowThreads - 1) / kRowThreads, m), dim3(kRowThreads), 0, table, tokens, pos_table, x, x0, width, ld,
                          vocab, max_positions, scale, dev_dyn(l));
}

cudaError_t launch_scalar_norm_rows(const Launch& l, DenseType type, const float* x, const int32_t* rows, void* out, int width, int ld, int m, float gain, float eps) {
    if (width <= 0 || ld < width || ld % 4 || m <= 0) return cudaErrorInvalidValue;
    const dim3 grid((m + kRowThreads / 32 - 1) / (kRowThreads / 32)), block(kRowThreads);
    return type == kDenseF32 ? launch_chained(l, scalar_norm_rows_kernel<float>, grid, block, 0, x, rows, (float*)out, width, ld, m, gain, eps, dev_dyn(l))
                             : launch_chained(l, scalar_norm_rows_kernel<bf16>, grid, block, 0, x, rows, (bf16*)out, width, ld, m, gain, eps, dev_dyn(l));
}

cudaError_t launch_pair_rows(const Launch& l, DenseType type, const float* x, const float* x0, void* out, int ld, int m) {
    if (ld <= 0 || m <= 0) return cudaErrorInvalidValue;
    const dim3 grid((2 * ld + kRowThreads - 1) / kRowThreads, m), block(kRowThreads);
    return type == kDenseF32 ? launch_chained(l, pair_rows_kernel<float>, grid, block, 0, x, x0, (float*)out, ld, dev_dyn(l))
                             : launch_chained(l, pair_rows_kernel<bf16>, grid, block, 0, x, x0, (bf16*)out, ld, dev_dyn(l));
}

cudaError_t launch_argmax_f32_partials(const Launch& l, const float* logits, uint64_t* partials, int vocab, int chunk, int rows) {
    if (vocab <= 0 || chunk <= 0 || rows <= 0) return cudaErrorInvalidValue;
    return launch_chained(l, argmax_f32_partials_kernel, dim3((vocab + chunk - 1) / chunk, rows), dim3(kRowThreads), 0, logits, partials, vocab, chunk, dev_dyn(l));
}

}  // namespace smelt
