// Row kernels of the prompt chunks of mixer / feed-forward stacks: embedding, the residual sum with
// its two norms, the routing of a chunk's tokens to experts and back.
#include <algorithm>

#include "stack.h"

namespace smelt {

namespace {

constexpr int kRowThreads = 256;

__global__ void __launch_bounds__(kRowThreads) embed_rows_kernel(const bf16* table, const int32_t* tokens, float* x, int width, int ld, uint32_t vocab, float scale, DevDyn dyn) {
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(dyn)) return;
    const uint32_t r = blockIdx.y, tok = (uint32_t)tokens[r];
    const int i = blockIdx.x * kRowThreads + threadIdx.x;
    if (i >= width || tok >= vocab) return;  // the host validates the ids
    x[(size_t)r * ld + i] = to_f32(table[(size_t)tok * width + i]) * scale;
}

__device__ __forceinline__ float4 ld_bf16x4(const bf16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xFFFF0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xFFFF0000u));
}
__device__ __forceinline__ float sumsq4(const float4& v, float ss) { return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss)))); }
template <class T> __device__ __forceinline__ void store4(T* dst, const float4& v) {
    if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(dst) = v;
    } else {
        const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
        *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
    }
}

// The sum over a CTA of kRowThreads, the same in every thread; scratch: eight floats used once.
__device__ __forceinline__ float row_sum(float v, float* scratch) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < kRowThreads / 32; ++w) tot += scratch[w];
    return tot;
}

// One CTA per row; N: float4s a thread keeps in registers (rows longer than N * 1024 are read again).
template <class T, int N>
__global__ void __launch_bounds__(kRowThreads) residual_norm_rows_kernel(const ResidualNormArgs a) {
    __shared__ float scratch[2][kRowThreads / 32];
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    const int r = blockIdx.x, src = a.rows ? a.rows[r] : r, n4 = a.ld / 4;
    float4* x = reinterpret_cast<float4*>(a.x + (size_t)src * a.ld);
    const float4* y = a.y ? reinterpret_cast<const float4*>(a.y + (size_t)src * a.ld) : nullptr;
    float4 s[N];
    float fy = 0.f, ss = 0.f;
    if (y) {
        float4 yv[N];
#pragma unroll
        for (int j = 0; j < N; ++j) {
            const int i = threadIdx.x + j * kRowThreads;
            yv[j] = i < n4 ? y[i] : make_float4(0.f, 0.f, 0.f, 0.f);
            s[j] = i < n4 ? x[i] : make_float4(0.f, 0.f, 0.f, 0.f);
            ss = sumsq4(yv[j], ss);
        }
        for (int i = threadIdx.x + N * kRowThreads; i < n4; i += kRowThreads) ss = sumsq4(y[i], ss);
        fy = rsqrtf(row_sum(ss, scratch[0]) / (float)a.width + a.eps);
        auto add = [&](float4& v, const float4& b, int i) {
            const float4 w = ld_bf16x4(a.post_w + 4 * i);
            v.x = fmaf(b.x * fy, 1.f + w.x, v.x);
            v.y = fmaf(b.y * fy, 1.f + w.y, v.y);
            v.z = fmaf(b.z * fy, 1.f + w.z, v.z);
            v.w = fmaf(b.w * fy, 1.f + w.w, v.w);
        };
        ss = 0.f;
#pragma unroll
        for (int j = 0; j < N; ++j) {
            const int i = threadIdx.x + j * kRowThreads;
            if (i >= n4) continue;
            add(s[j], yv[j], i);
            ss = sumsq4(s[j], ss);
            if (!a.rows) x[i] = s[j];
        }
        for (int i = threadIdx.x + N * kRowThreads; i < n4; i += kRowThreads) {
            float4 v = x[i];
            add(v, y[i], i);
            ss = sumsq4(v, ss);
            if (!a.rows) x[i] = v;
        }
    } else {
#pragma unroll
        for (int j = 0; j < N; ++j) {
            const int i = threadIdx.x + j * kRowThreads;
            s[j] = i < n4 ? x[i] : make_float4(0.f, 0.f, 0.f, 0.f);
            ss = sumsq4(s[j], ss);
        }
        for (int i = threadIdx.x + N * kRowThreads; i < n4; i += kRowThreads) ss = sumsq4(x[i], ss);
    }
    const float f = rsqrtf(row_sum(ss, scratch[1]) / (float)a.width + a.eps);
    T* out = static_cast<T*>(a.out) + (size_t)r * a.ld;
    auto emit = [&](const float4& v, int i) {
        const float4 w = ld_bf16x4(a.norm_w + 4 * i);
        const float4 h = make_float4(v.x * f * (1.f + w.x), v.y * f * (1.f + w.y), v.z * f * (1.f + w.z), v.w * f * (1.f + w.w));
        store4(out + 4 * i, h);
        if (a.h_f32) *reinterpret_cast<float4*>(a.h_f32 + (size_t)r * a.ld + 4 * i) = h;
    };
#pragma unroll
    for (int j = 0; j < N; ++j) {
        const int i = threadIdx.x + j * kRowThreads;
        if (i < n4) emit(s[j], i);
    }
    for (int i = threadIdx.x + N * kRowThreads; i < n4; i += kRowThreads) {
        float4 v = x[i];
        if (y && a.rows) {  // the sum was not written back
            const float4 b = y[i], w = ld_bf16x4(a.post_w + 4 * i);
            v = make_float4(fmaf(b.x * fy, 1.f + w.x, v.x), fmaf(b.y * fy, 1.f + w.y, v.y), fmaf(b.z * fy, 1.f + w.z, v.z), fmaf(b.w * fy, 1.f + w.w, v.w));
        }
        emit(v, i);
    }
}

template <class T>
cudaError_t residual_norm_t(const Launch& l, const ResidualNormArgs& a) {
    const dim3 grid(a.m), block(kRowThreads);
    if (a.ld <= 1024) return launch_chained(l, residual_norm_rows_kernel<T, 1>, grid, block, 0, a);
    if (a.ld <= 2048) return launch_chained(l, residual_norm_rows_kernel<T, 2>, grid, block, 0, a);
    if (a.ld <= 4096) return launch_chained(l, residual_norm_rows_kernel<T, 4>, grid, block, 0, a);
    return launch_chained(l, residual_norm_rows_kernel<T, 8>, grid, block, 0, a);
}

// ── experts ─────────────────────────────────────────────────────────────────
// One warp per token: the `top` largest logits (ties to the lower index) and the softmax over them.
__global__ void __launch_bounds__(kRowThreads) moe_choose_kernel(const MoeArgs a) {
    extern __shared__ float s_logits[];  // [warps][experts]
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * (kRowThreads / 32) + warp;
    if (t >= a.m) return;
    float* sl = s_logits + (size_t)warp * a.experts;
    for (int e = lane; e < a.experts; e += 32) sl[e] = a.logits[(size_t)t * a.experts + e];
    __syncwarp();
    float first = 0.f, total = 0.f;
    int2* chosen = a.chosen + (size_t)t * a.top;
    for (int n = 0; n < a.top; ++n) {
        float v = -INFINITY;
        int at = a.experts;
        for (int e = lane; e < a.experts; e += 32)
            if (sl[e] > v || at == a.experts) { v = sl[e]; at = e; }
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, v, o);
            const int oa = __shfl_xor_sync(0xffffffffu, at, o);
            if (oa < a.experts && (at == a.experts || ov > v || (ov == v && oa < at))) { v = ov; at = oa; }
        }
        if (n == 0) first = v;
        const float p = expf(v - first);
        total += p;
        if (lane == 0) {
            chosen[n] = make_int2(at, __float_as_int(p));
            sl[at] = -INFINITY;
        }
        __syncwarp();
    }
    for (int n = lane; n < a.top; n += 32) chosen[n].y = __float_as_int(__int_as_float(chosen[n].y) / total);
}

// One CTA: rows of the permuted chunk, expert after expert, and the table of row tiles.
constexpr int kPlaceThreads = 1024;
__global__ void __launch_bounds__(kPlaceThreads) moe_place_kernel(const MoeArgs a) {
    extern __shared__ int s_int[];  // counts, then next rows; first rows; first entries
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    int *next = s_int, *first = next + a.experts;
    const int tid = threadIdx.x, pairs = a.m * a.top;
    for (int e = tid; e < a.experts; e += kPlaceThreads) next[e] = 0;
    __syncthreads();
    for (int i = tid; i < pairs; i += kPlaceThreads) atomicAdd(&next[a.chosen[i].x], 1);
    __syncthreads();
    if (tid < 32) {  // exclusive sums over the experts, 32 at a time
        int rows = 0, entries = 0;
        for (int e0 = 0; e0 < a.experts; e0 += 32) {
            const int e = e0 + tid, n = e < a.experts ? next[e] : 0, tiles = (n + a.tile - 1) / a.tile;
            int rs = n, es = tiles;
            for (int o = 1; o < 32; o <<= 1) {
                const int r2 = __shfl_up_sync(0xffffffffu, rs, o), e2 = __shfl_up_sync(0xffffffffu, es, o);
                if (tid >= o) { rs += r2; es += e2; }
            }
            if (e < a.experts) {
                first[e] = rows + rs - n;
                for (int k = 0; k < tiles; ++k) a.table[1 + entries + es - tiles + k] = make_int4(e, first[e] + k * a.tile, min(a.tile, n - k * a.tile), 0);
            }
            rows += __shfl_sync(0xffffffffu, rs, 31);
            entries += __shfl_sync(0xffffffffu, es, 31);
        }
        if (tid == 0) a.table[0] = make_int4(entries, 0, 0, 0);
    }
    __syncthreads();
    for (int e = tid; e < a.experts; e += kPlaceThreads) next[e] = first[e];
    __syncthreads();
    for (int i = tid; i < pairs; i += kPlaceThreads) a.place[i] = atomicAdd(&next[a.chosen[i].x], 1);
}

// A token's activations into the rows of its experts; 16 bytes a thread.
__global__ void __launch_bounds__(kRowThreads) moe_gather_kernel(const MoeArgs a, int row16) {
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    const int t = blockIdx.x;
    const uint4* src = static_cast<const uint4*>(a.h) + (size_t)t * row16;
    for (int n = 0; n < a.top; ++n) {
        uint4* dst = static_cast<uint4*>(a.permuted) + (size_t)a.place[(size_t)t * a.top + n] * row16;
        for (int i = threadIdx.x; i < row16; i += kRowThreads) dst[i] = src[i];
    }
}

__global__ void __launch_bounds__(kRowThreads) moe_combine_kernel(const MoeArgs a) {
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    const int t = blockIdx.x;
    for (int i = threadIdx.x; i < a.ld / 4; i += kRowThreads) {
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int n = 0; n < a.top; ++n) {
            const float w = __int_as_float(a.chosen[(size_t)t * a.top + n].y);
            const float4 v = *reinterpret_cast<const float4*>(a.y_rows + (size_t)a.place[(size_t)t * a.top + n] * a.ld + 4 * i);
            acc.x = fmaf(w, v.x, acc.x); acc.y = fmaf(w, v.y, acc.y); acc.z = fmaf(w, v.z, acc.z); acc.w = fmaf(w, v.w, acc.w);
        }
        *reinterpret_cast<float4*>(a.y + (size_t)t * a.ld + 4 * i) = acc;
    }
}

bool bad(const MoeArgs& a) { return a.m <= 0 || a.experts <= 0 || a.experts > 4096 || a.top <= 0 || a.top > kMaxTop || a.top > a.experts; }

}  // namespace

cudaError_t launch_embed_rows(const Launch& l, const bf16* table, const int32_t* tokens, float* x, int width, int ld, int m, uint32_t vocab, float scale) {
    if (width <= 0 || ld < width || m <= 0) return cudaErrorInvalidValue;
    return launch_chained(l, embed_rows_kernel, dim3((width + kRowThreads - 1) / kRowThreads, m), dim3(kRowThreads), 0, table, tokens, x, width, ld, vocab, scale, dev_dyn(l));
}

cudaError_t launch_residual_norm_rows(const Launch& l, DenseType type, ResidualNormArgs a) {
    if (a.width <= 0 || a.ld < a.width || a.ld % 4 || a.m <= 0) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    return type == kDenseF32 ? residual_norm_t<float>(l, a) : residual_norm_t<bf16>(l, a);
}

cudaError_t launch_moe_route(const Launch& l, MoeArgs a) {
    if (bad(a) || a.tile <= 0) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    const int warps = kRowThreads / 32;
    cudaError_t e = launch_chained(l, moe_choose_kernel, dim3((a.m + warps - 1) / warps), dim3(kRowThreads), (size_t)warps * a.experts * sizeof(float), a);
    return e == cudaSuccess ? launch_chained(l, moe_place_kernel, dim3(1), dim3(kPlaceThreads), (size_t)2 * a.experts * sizeof(int), a) : e;
}

cudaError_t launch_moe_gather(const Launch& l, DenseType type, MoeArgs a) {
    if (bad(a) || a.ld % 8) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    return launch_chained(l, moe_gather_kernel, dim3(a.m), dim3(kRowThreads), 0, a, type == kDenseF32 ? a.ld / 4 : a.ld / 8);
}

cudaError_t launch_moe_combine(const Launch& l, MoeArgs a) {
    if (bad(a) || a.ld % 4) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    return launch_chained(l, moe_combine_kernel, dim3(a.m), dim3(kRowThreads), 0, a);
}

}  // namespace smelt
