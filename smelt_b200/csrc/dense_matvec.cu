// Matrix-vector product with bf16 weights for one decoded token.
//
// The activation row is staged once per CTA in fp32 (a decode step keeps all its activations in
// fp32, so the only 16-bit operand is the stored weight) and, where the layer's norm is one
// number, the norm is one factor per row that the epilogue applies.  The weight stream
// (matvec.cuh) starts ahead of the wait for the launch in front, which the weights do not depend on.
#include "matvec.cuh"

namespace smelt {

namespace {

using namespace matvec;

template <int MODE>
__global__ void __launch_bounds__(kThreads, 1) dense_matvec_kernel(const DenseMatvecArgs a, int rows_per_cta, int ks) {
    extern __shared__ __align__(16) float smem[];
    const int chunks = (a.cols + kChunkCols - 1) / kChunkCols;
    float* sx = smem;
    float* part = smem + (size_t)chunks * kChunkCols;
    __shared__ float s_sum[kWarps];
    const int tid = threadIdx.x;
    const int r0 = blockIdx.x * rows_per_cta, r1 = min(a.rows, r0 + rows_per_cta);
    float factor = 1.f;
    const bool done = stream_rows<true>(MatrixRows{a.w, a.cols}, r0, r1, a.cols, chunks, ks, sx, part, [&] {
        pdl_wait();
        if (dyn_skip(a.dyn)) return false;
        float ss = 0.f;
#pragma unroll 4
        for (int i = tid * 4; i < chunks * kChunkCols; i += kThreads * 4) {
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (i < a.cols) v = *reinterpret_cast<const float4*>(a.xb && i >= a.ka ? a.xb + (i - a.ka) : a.xa + i);
            ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
            *reinterpret_cast<float4*>(sx + staged(i)) = v;
        }
        if (a.norm) {
            ss = warp_sum(ss);
            if ((tid & 31) == 0) s_sum[tid >> 5] = ss;
        }
        __syncthreads();
        if (a.norm) {
            float tot = 0.f;
#pragma unroll
            for (int w = 0; w < kWarps; ++w) tot += s_sum[w];
            factor = a.gain * rsqrtf(tot / (float)a.width + a.eps);
        }
        return true;
    });
    if (!done) return;
    for (int i = tid; i < r1 - r0; i += kThreads) {
        const float v = sum_parts(part, i, ks) * factor;
        const int row = r0 + i;
        if (MODE == kDenseAddF32) static_cast<float*>(a.out.y0)[row] += v;
        else if (row < a.out.split) static_cast<float*>(a.out.y0)[row] = v;
        else static_cast<float*>(a.out.y1)[row - a.out.split] = xielu(v, a.out.rising, a.out.falling);
    }
}

}  // namespace

cudaError_t launch_dense_matvec(const Launch& l, int mode, DenseMatvecArgs a) {
    if (a.rows <= 0 || a.cols <= 0 || a.cols % 64 || (a.xb && a.ka % 4) || (mode == kDenseAddF32 && a.out.split != a.rows)) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    const Split s = split_rows(a.rows, a.cols, a.sm_count);
    const int grid = (a.rows + s.rows_per_cta - 1) / s.rows_per_cta;
    if (s.smem() > kMaxShared) return cudaErrorInvalidValue;
    return mode == kDenseAddF32 ? launch_chained(l, dense_matvec_kernel<kDenseAddF32>, dim3(grid), dim3(kThreads), s.smem(), a, s.rows_per_cta, s.ks)
                                : launch_chained(l, dense_matvec_kernel<kDenseStoreF32>, dim3(grid), dim3(kThreads), s.smem(), a, s.rows_per_cta, s.ks);
}

}  // namespace smelt
