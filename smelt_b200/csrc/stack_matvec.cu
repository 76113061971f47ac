// Matrix-vector products of one decoded token, fused with what stands in front of and behind them:
// the residual sum with the norm after the last sublayer, the norm before this one, the token
// shift and its mixes, the choice of experts, bias and activation.
//
// A norm over the whole row needs every CTA's part of the product before it, so each CTA of the
// next product forms it anew while it stages its activation row; CTA 0 writes the residual row to
// the other one of two buffers.  The norm that a plain matrix follows is one factor in the
// epilogue, its weight is applied while staging.  The weight stream (matvec.cuh) starts ahead of
// the wait for the launch in front, except where the experts are chosen by it.
#include <algorithm>

#include "matvec.cuh"
#include "stack.h"

namespace smelt {

namespace {

using namespace matvec;

__device__ __forceinline__ float4 ld_bf16x4(const bf16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xFFFF0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xFFFF0000u));
}
__device__ __forceinline__ float sumsq4(const float4& v, float ss) { return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss)))); }

// One warp: the `top` largest of sl[0 .. experts) (ties to the lower index) and the softmax over them; sl is consumed.
__device__ __forceinline__ void choose_experts(float* sl, int experts, int top, int* s_expert, float* s_weight, int lane) {
    float best_of_all = 0.f, total = 0.f;
    for (int n = 0; n < top; ++n) {
        float v = -INFINITY;
        int at = experts;
        for (int e = lane; e < experts; e += 32)
            if (sl[e] > v || at == experts) { v = sl[e]; at = e; }
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, v, o);
            const int oa = __shfl_xor_sync(0xffffffffu, at, o);
            if (oa < experts && (at == experts || ov > v || (ov == v && oa < at))) { v = ov; at = oa; }
        }
        if (n == 0) best_of_all = v;
        const float p = expf(v - best_of_all);
        total += p;
        if (lane == 0) {
            s_expert[n] = at;
            s_weight[n] = p;
            sl[at] = -INFINITY;
        }
        __syncwarp();
    }
    for (int n = lane; n < top; n += 32) s_weight[n] /= total;
    __syncwarp();
}

// Rows of one matrix, or of the chosen experts' matrices (of rows x cols each): one behind the other, or side by side.
template <int IN>
struct Rows : MatrixRows {
    __device__ __forceinline__ Rows(const StackMatvecArgs& a, const int*) : MatrixRows{a.w, a.cols} {}
};
template <>
struct Rows<kInExpertsIn> {
    const bf16* w;
    int rows, cols;
    const int* expert;
    struct Pairs { const uint4 *low, *high; };
    __device__ __forceinline__ Rows(const StackMatvecArgs& a, const int* expert) : w(a.w), rows(a.rows), cols(a.cols), expert(expert) {}
    __device__ __forceinline__ const uint4* at(int row, int col) const {
        const int n = min(row / rows, kMaxTop - 1);  // rows past the last expert's are not read
        return reinterpret_cast<const uint4*>(w + ((size_t)expert[n] * rows + (row - n * rows)) * cols + col);
    }
    __device__ __forceinline__ Pairs first(int row, int col) const { return {at(row, col), at(row + 2, col)}; }  // an even number of rows an expert: a pair is never divided
    __device__ __forceinline__ const uint4* after(const Pairs& p, int r) const { return (r < 2 ? p.low : p.high) + (r & 1) * (cols / 8); }
};
template <>
struct Rows<kInExpertsOut> {
    const bf16* w;
    int rows, cols;
    const int* expert;
    __device__ __forceinline__ Rows(const StackMatvecArgs& a, const int* expert) : w(a.w), rows(a.rows), cols(a.cols), expert(expert) {}
    __device__ __forceinline__ const uint4* first(int row, int col) const {
        const int n = min(col / cols, kMaxTop - 1);  // columns past the last expert's are not read
        return reinterpret_cast<const uint4*>(w + ((size_t)expert[n] * rows + row) * cols + (col - n * cols));
    }
    __device__ __forceinline__ const uint4* after(const uint4* p, int r) const { return p + (size_t)r * (cols / 8); }
};

template <int IN>
__global__ void __launch_bounds__(kThreads, 1) stack_matvec_kernel(const StackMatvecArgs a, int rows_per_cta, int ks) {
    extern __shared__ __align__(16) float smem[];
    constexpr bool kSelect = IN == kInExpertsIn || IN == kInExpertsOut;
    const int cols = IN == kInExpertsOut ? a.cols * a.top : a.cols, chunks = (cols + kChunkCols - 1) / kChunkCols;
    float* sx = smem;
    float* part = smem + (size_t)chunks * kChunkCols;
    __shared__ float s_sum[2][kWarps];
    __shared__ int s_expert[kMaxTop];
    __shared__ float s_weight[kMaxTop];
    const int tid = threadIdx.x;
    int r0 = blockIdx.x * rows_per_cta, r1 = min(IN == kInExpertsIn ? a.rows * a.top : a.rows, r0 + rows_per_cta), group = 0;
    if (IN == kInShift) {  // a CTA's rows belong to one group
        const int per_group = (a.group_rows + rows_per_cta - 1) / rows_per_cta;
        group = min((int)blockIdx.x / per_group, kMixes - 1);
        r0 = group * a.group_rows + ((int)blockIdx.x - group * per_group) * rows_per_cta;
        r1 = min(group == kMixes - 1 ? a.rows : (group + 1) * a.group_rows, r0 + rows_per_cta);
    }
    float factor = 1.f;
    const bool done = stream_rows<!kSelect>(Rows<IN>(a, s_expert), r0, r1, cols, chunks, ks, sx, part, [&] {
        pdl_wait();
        if (dyn_skip(a.dyn)) return false;
        const int staged_cols = chunks * kChunkCols;
        if (IN == kInExpertsIn) {
            float* sl = part + (size_t)rows_per_cta * ks;  // [experts]
            for (int i = tid; i < a.experts; i += kThreads) sl[i] = a.logits[i];
            __syncthreads();
            if (tid < 32) {
                choose_experts(sl, a.experts, a.top, s_expert, s_weight, tid);
                if (blockIdx.x == 0)
                    for (int n = tid; n < a.top; n += 32) a.chosen[n] = make_int2(s_expert[n], __float_as_int(s_weight[n]));
            }
        } else if (IN == kInExpertsOut) {
            if (tid < a.top) s_expert[tid] = a.chosen[tid].x;
        }
        if (IN == kInPlain || kSelect) {
#pragma unroll 4
            for (int i = tid * 4; i < staged_cols; i += kThreads * 4)
                *reinterpret_cast<float4*>(sx + staged(i)) = i < cols ? *reinterpret_cast<const float4*>(a.x + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            __syncthreads();
        } else if (IN == kInNorm) {
            float ss = 0.f;
#pragma unroll 4
            for (int i = tid * 4; i < staged_cols; i += kThreads * 4) {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                if (i < cols) {
                    v = *reinterpret_cast<const float4*>(a.x + i);
                    ss = sumsq4(v, ss);
                    const float4 w = ld_bf16x4(a.norm_w + i);
                    v = make_float4(v.x * w.x, v.y * w.y, v.z * w.z, v.w * w.w);
                }
                *reinterpret_cast<float4*>(sx + staged(i)) = v;
            }
            factor = rsqrtf(cta_sum(ss, s_sum[0]) / (float)a.width + a.eps);
        } else {
            float fy = 0.f;
            if (a.y) {
                float ss = 0.f;
#pragma unroll 4
                for (int i = tid * 4; i < cols; i += kThreads * 4) {
                    const float4 v = *reinterpret_cast<const float4*>(a.y + i);
                    ss = sumsq4(v, ss);
                    *reinterpret_cast<float4*>(sx + staged(i)) = v;  // read again by this thread only
                }
                fy = rsqrtf(cta_sum(ss, s_sum[0]) / (float)a.width + a.eps);
            }
            float ss = 0.f;
#pragma unroll 4
            for (int i = tid * 4; i < staged_cols; i += kThreads * 4) {
                float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
                if (i < cols) {
                    s = *reinterpret_cast<const float4*>(a.x + i);
                    if (a.y) {
                        const float4 y = *reinterpret_cast<const float4*>(sx + staged(i)), w = ld_bf16x4(a.post_w + i);
                        s.x = fmaf(y.x * fy, 1.f + w.x, s.x);
                        s.y = fmaf(y.y * fy, 1.f + w.y, s.y);
                        s.z = fmaf(y.z * fy, 1.f + w.z, s.z);
                        s.w = fmaf(y.w * fy, 1.f + w.w, s.w);
                        if (blockIdx.x == 0 && a.x_out) *reinterpret_cast<float4*>(a.x_out + i) = s;
                    }
                    ss = sumsq4(s, ss);
                    const float4 w = ld_bf16x4(a.norm_w + i);
                    s = make_float4(s.x * (1.f + w.x), s.y * (1.f + w.y), s.z * (1.f + w.z), s.w * (1.f + w.w));
                }
                *reinterpret_cast<float4*>(sx + staged(i)) = s;
            }
            factor = rsqrtf(cta_sum(ss, s_sum[1]) / (float)a.width + a.eps);
            const bool store_h = a.h_out && blockIdx.x == 0;
            if (IN == kInShift || store_h) {
                const bool has_before = IN == kInShift && dyn_position(a.dyn) != 0u;
                const bf16* mu = IN == kInShift ? a.mu + (size_t)group * a.cols : nullptr;
#pragma unroll 4
                for (int i = tid * 4; i < cols; i += kThreads * 4) {
                    float4* at = reinterpret_cast<float4*>(sx + staged(i));
                    float4 h = *at;
                    h = make_float4(h.x * factor, h.y * factor, h.z * factor, h.w * factor);
                    if (store_h) *reinterpret_cast<float4*>(a.h_out + i) = h;
                    if (IN == kInShift) {
                        const float4 b = has_before ? *reinterpret_cast<const float4*>(a.before + i) : make_float4(0.f, 0.f, 0.f, 0.f), t = ld_bf16x4(mu + i);
                        *at = make_float4(fmaf(b.x - h.x, t.x, h.x), fmaf(b.y - h.y, t.y, h.y), fmaf(b.z - h.z, t.z, h.z), fmaf(b.w - h.w, t.w, h.w));
                    }
                }
            }
            if (IN == kInShift) {
                factor = 1.f;
                __syncthreads();
            }
        }
        return true;
    });
    if (!done) return;
    if (IN == kInExpertsIn) {  // pairs of rows: gate, up
        for (int i = tid; i < (r1 - r0) / 2; i += kThreads)
            a.out[r0 / 2 + i] = clamped_glu(sum_parts(part, 2 * i, ks), sum_parts(part, 2 * i + 1, ks), a.limit) * s_weight[(r0 + 2 * i) / a.rows];
    } else {
        for (int i = tid; i < r1 - r0; i += kThreads) {
            const int row = r0 + i;
            float v = sum_parts(part, i, ks) * factor;
            if (a.bias) v += to_f32(a.bias[row]);
            if (a.act == kActRelu2) { v = fmaxf(v, 0.f); v *= v; }
            a.out[row] = v;
        }
    }
}

}  // namespace

cudaError_t launch_stack_matvec(const Launch& l, int input, StackMatvecArgs a) {
    if (a.rows <= 0 || a.cols <= 0 || a.cols % 64 || a.width > a.cols) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    const bool experts = input == kInExpertsIn || input == kInExpertsOut;
    if (experts && (a.top <= 0 || a.top > kMaxTop || a.top > a.experts || (input == kInExpertsIn && a.rows % 2))) return cudaErrorInvalidValue;
    const int rows = input == kInExpertsIn ? a.rows * a.top : a.rows, cols = input == kInExpertsOut ? a.cols * a.top : a.cols;
    Split s = split_rows(rows, cols, a.sm_count);
    if (input == kInExpertsIn) s.rows_per_cta = (s.rows_per_cta + 1) / 2 * 2;  // a pair stays in one CTA
    int grid = (rows + s.rows_per_cta - 1) / s.rows_per_cta;
    if (input == kInShift) {
        const int last = rows - (kMixes - 1) * a.group_rows;
        if (a.group_rows <= 0 || last <= 0 || !a.mu || !a.before) return cudaErrorInvalidValue;
        const int sm = a.sm_count > 0 ? a.sm_count : 148;
        auto ctas = [&](int per) { return (kMixes - 1) * ((a.group_rows + per - 1) / per) + (last + per - 1) / per; };
        while (ctas(s.rows_per_cta) > sm && s.rows_per_cta < std::max(a.group_rows, last)) ++s.rows_per_cta;
        grid = ctas(s.rows_per_cta);
    }
    const size_t smem = s.smem() + (input == kInExpertsIn ? (size_t)a.experts * sizeof(float) : 0);
    if (smem > kMaxShared) return cudaErrorInvalidValue;
    switch (input) {
        case kInPlain: return launch_chained(l, stack_matvec_kernel<kInPlain>, dim3(grid), dim3(kThreads), smem, a, s.rows_per_cta, s.ks);
        case kInNorm: return launch_chained(l, stack_matvec_kernel<kInNorm>, dim3(grid), dim3(kThreads), smem, a, s.rows_per_cta, s.ks);
        case kInResidual: return launch_chained(l, stack_matvec_kernel<kInResidual>, dim3(grid), dim3(kThreads), smem, a, s.rows_per_cta, s.ks);
        case kInShift: return launch_chained(l, stack_matvec_kernel<kInShift>, dim3(grid), dim3(kThreads), smem, a, s.rows_per_cta, s.ks);
        case kInExpertsIn: return launch_chained(l, stack_matvec_kernel<kInExpertsIn>, dim3(grid), dim3(kThreads), smem, a, s.rows_per_cta, s.ks);
        case kInExpertsOut: return launch_chained(l, stack_matvec_kernel<kInExpertsOut>, dim3(grid), dim3(kThreads), smem, a, s.rows_per_cta, s.ks);
        default: return cudaErrorInvalidValue;
    }
}

}  // namespace smelt
