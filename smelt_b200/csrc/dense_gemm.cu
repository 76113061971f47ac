// Matrix products of a prompt chunk: Y[m, rows] = X[m, cols] . W[rows, cols]^T, bf16 weights.
//
// gemm_f32_kernel: fp32 activations and arithmetic on the CUDA cores (the fp32 table).
#include <algorithm>

#include "dense.h"

namespace smelt {

namespace {

template <int MODE, class T>
__device__ __forceinline__ void dense_store(const DenseOut& o, int token, int row, float v) {
    if (MODE == kDenseStoreF32) static_cast<float*>(o.y0)[(size_t)token * o.ld0 + row] = v;
    else if (MODE == kDenseAddF32) static_cast<float*>(o.y0)[(size_t)token * o.ld0 + row] += v;
    else if (row < o.split) static_cast<T*>(o.y0)[(size_t)token * o.ld0 + row] = from_f32<T>(v);
    else static_cast<T*>(o.y1)[(size_t)token * o.ld1 + (row - o.split)] = from_f32<T>(xielu(v, o.rising, o.falling));
}

constexpr int kTile = 64, kStep = 32;

template <int MODE, class T>
__global__ void __launch_bounds__(256) gemm_f32_kernel(const DenseGemmArgs a, DevDyn dyn) {
    __shared__ float xs[kTile][kStep + 1], ws[kTile][kStep + 1];
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(dyn)) return;
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int n0 = blockIdx.x * kTile, m0 = blockIdx.y * kTile;
    const T* x = static_cast<const T*>(a.x);
    float acc[4][4] = {};
    for (int k0 = 0; k0 < a.cols; k0 += kStep) {
        for (int i = tid; i < kTile * kStep; i += 256) {
            const int r = i / kStep, c = i % kStep;
            xs[r][c] = m0 + r < a.m ? to_f32(x[(size_t)(m0 + r) * a.cols + k0 + c]) : 0.f;
            ws[r][c] = n0 + r < a.rows ? to_f32(a.w[(size_t)(n0 + r) * a.cols + k0 + c]) : 0.f;
        }
        __syncthreads();
#pragma unroll 8
        for (int k = 0; k < kStep; ++k) {
            float xv[4], wv[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { xv[i] = xs[ty + 16 * i][k]; wv[i] = ws[tx + 16 * i][k]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if (m0 + ty + 16 * i < a.m && n0 + tx + 16 * j < a.rows) dense_store<MODE, T>(a.out, m0 + ty + 16 * i, n0 + tx + 16 * j, acc[i][j]);
}

template <class T>
cudaError_t launch_f32(const Launch& l, int mode, const DenseGemmArgs& a) {
    const dim3 grid((a.rows + kTile - 1) / kTile, (a.m + kTile - 1) / kTile), block(256);
    switch (mode) {
        case kDenseStoreF32: return launch_chained(l, gemm_f32_kernel<kDenseStoreF32, T>, grid, block, 0, a, dev_dyn(l));
        case kDenseAddF32: return launch_chained(l, gemm_f32_kernel<kDenseAddF32, T>, grid, block, 0, a, dev_dyn(l));
        case kDenseStoreAct: return launch_chained(l, gemm_f32_kernel<kDenseStoreAct, T>, grid, block, 0, a, dev_dyn(l));
        default: return cudaErrorInvalidValue;
    }
}

}  // namespace

cudaError_t launch_dense_gemm(const Launch& l, DenseType type, int mode, const DenseGemmArgs& a) {
    if (a.rows <= 0 || a.cols <= 0 || a.cols % 64 || a.m <= 0 || (mode != kDenseStoreAct && a.out.split != a.rows)) return cudaErrorInvalidValue;
    return type == kDenseF32 ? launch_f32<float>(l, mode, a) : launch_f32<bf16>(l, mode, a);
}

}  // namespace smelt
