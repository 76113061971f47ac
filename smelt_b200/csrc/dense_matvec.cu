// Matrix-vector product with bf16 weights for one decoded token.
//
// The activation row is staged once per CTA in fp32 (a decode step keeps all its activations in
// fp32, so the only 16-bit operand is the stored weight) and, where the layer's norm is one
// number, the norm is one factor per row that the epilogue applies.  One CTA per SM owns a
// contiguous range of rows; its sixteen warps form 16 / KS row groups of KS warps that split the
// columns.  A warp's work is a sequence of items of four rows x 256 columns, so that every
// activation value read from shared memory feeds four weights; kDepth items are in flight in
// registers (256 bytes a lane), across the end of a group of rows and, at the start, across the
// wait for the launch in front, which the weights do not depend on.  Partial sums meet in shared
// memory once per CTA and are added in warp order.
#include <algorithm>

#include "dense.h"

namespace smelt {

namespace {

constexpr int kThreads = 512, kWarps = 16, kRowsPerPass = 4, kChunkCols = 256, kDepth = 4;

__device__ __forceinline__ uint4 ld_stream(const uint4* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}

__device__ __forceinline__ float dot8(const uint4& w, const float4& a, const float4& b, float acc) {
    const uint32_t u[4] = {w.x, w.y, w.z, w.w};
    const float x[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        acc = fmaf(__uint_as_float(u[i] << 16), x[2 * i], acc);
        acc = fmaf(__uint_as_float(u[i] & 0xFFFF0000u), x[2 * i + 1], acc);
    }
    return acc;
}

// The sums of four values over the warp; the lane gets the one of row 2 (lane bit 4) + (lane bit 3).
__device__ __forceinline__ float sum_four_rows(const float (&v)[kRowsPerPass], int lane) {
    const bool up = lane & 16, odd = lane & 8;
    const float k0 = (up ? v[2] : v[0]) + __shfl_xor_sync(0xffffffffu, up ? v[0] : v[2], 16);
    const float k1 = (up ? v[3] : v[1]) + __shfl_xor_sync(0xffffffffu, up ? v[1] : v[3], 16);
    float k = (odd ? k1 : k0) + __shfl_xor_sync(0xffffffffu, odd ? k0 : k1, 8);
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) k += __shfl_xor_sync(0xffffffffu, k, o);
    return k;
}

template <int MODE>
__global__ void __launch_bounds__(kThreads, 1) dense_matvec_kernel(const DenseMatvecArgs a, int rows_per_cta, int ks) {
    extern __shared__ __align__(16) float smem[];
    const int chunks = (a.cols + kChunkCols - 1) / kChunkCols;
    float* sx = smem;                          // [chunks][2][32][4]: a lane's eight values as two conflict-free halves
    float* part = smem + (size_t)chunks * kChunkCols;
    __shared__ float s_sum[kWarps];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int kid = warp % ks, group = warp / ks, step = kWarps / ks * kRowsPerPass;
    const int r0 = blockIdx.x * rows_per_cta, r1 = min(a.rows, r0 + rows_per_cta);
    pdl_trigger();

    struct Item { int row, chunk; };
    auto next = [&](Item& it) {
        it.chunk += ks;
        if (it.chunk >= chunks) { it.chunk = kid; it.row += step; }
    };
    auto load = [&](const Item& it, uint4 (&dst)[kRowsPerPass]) {
        const int col = it.chunk * kChunkCols + lane * 8;
        const uint4* p = reinterpret_cast<const uint4*>(a.w + (size_t)it.row * a.cols + col);
        const bool in = col < a.cols;
#pragma unroll
        for (int r = 0; r < kRowsPerPass; ++r) dst[r] = in && it.row + r < r1 ? ld_stream(p + (size_t)r * (a.cols / 8)) : make_uint4(0, 0, 0, 0);
    };
    uint4 buf[kDepth][kRowsPerPass];
    Item cur{r0 + group * kRowsPerPass, kid}, ahead = cur;
#pragma unroll
    for (int i = 0; i < kDepth; ++i) { load(ahead, buf[i]); next(ahead); }

    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    float ss = 0.f;
#pragma unroll 4
    for (int i = tid * 4; i < chunks * kChunkCols; i += kThreads * 4) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < a.cols) v = *reinterpret_cast<const float4*>(a.xb && i >= a.ka ? a.xb + (i - a.ka) : a.xa + i);
        ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
        const int c = i / kChunkCols, in = i % kChunkCols;
        *reinterpret_cast<float4*>(sx + c * kChunkCols + ((in >> 2) & 1) * 128 + (in >> 3) * 4) = v;
    }
    float factor = 1.f;
    if (a.norm) {
        ss = warp_sum(ss);
        if (lane == 0) s_sum[warp] = ss;
    }
    __syncthreads();
    if (a.norm) {
        float tot = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) tot += s_sum[w];
        factor = a.gain * rsqrtf(tot / (float)a.width + a.eps);
    }

    float acc[kRowsPerPass] = {0.f, 0.f, 0.f, 0.f};
    while (cur.row < r1) {
#pragma unroll
        for (int i = 0; i < kDepth; ++i) {
            if (cur.row >= r1) break;
            const float4 xa = *reinterpret_cast<const float4*>(sx + cur.chunk * kChunkCols + lane * 4);
            const float4 xb = *reinterpret_cast<const float4*>(sx + cur.chunk * kChunkCols + 128 + lane * 4);
#pragma unroll
            for (int r = 0; r < kRowsPerPass; ++r) acc[r] = dot8(buf[i][r], xa, xb, acc[r]);
            load(ahead, buf[i]);
            next(ahead);
            if (cur.chunk + ks >= chunks) {  // the last columns of these rows
                const float v = sum_four_rows(acc, lane);
                const int row = cur.row + (lane >> 4) * 2 + ((lane >> 3) & 1);
                if ((lane & 7) == 0 && row < r1) part[(size_t)(row - r0) * ks + kid] = v;
                acc[0] = acc[1] = acc[2] = acc[3] = 0.f;
            }
            next(cur);
        }
    }
    __syncthreads();
    for (int i = tid; i < r1 - r0; i += kThreads) {
        float v = 0.f;
        for (int k = 0; k < ks; ++k) v += part[(size_t)i * ks + k];
        v *= factor;
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
    const int sm = a.sm_count > 0 ? a.sm_count : 148;
    const int chunks = (a.cols + kChunkCols - 1) / kChunkCols;
    int ks = 1;
    while (ks < kWarps && ks * 2 <= chunks) ks *= 2;
    const size_t x_bytes = (size_t)chunks * kChunkCols * sizeof(float), limit = 225 * 1024;
    // one CTA per SM with an equal share of the rows, at least what keeps its row groups busy
    int rows_per_cta = (a.rows + sm - 1) / sm;
    rows_per_cta = std::max(rows_per_cta, std::min(kRowsPerPass * (kWarps / ks), 8));
    const int grid = (a.rows + rows_per_cta - 1) / rows_per_cta;
    const size_t smem = x_bytes + (size_t)rows_per_cta * ks * sizeof(float);
    if (smem > limit) return cudaErrorInvalidValue;
    return mode == kDenseAddF32 ? launch_chained(l, dense_matvec_kernel<kDenseAddF32>, dim3(grid), dim3(kThreads), smem, a, rows_per_cta, ks)
                                : launch_chained(l, dense_matvec_kernel<kDenseStoreF32>, dim3(grid), dim3(kThreads), smem, a, rows_per_cta, ks);
}

}  // namespace smelt
