// Matrix-vector product with bf16 weights for one decoded token.
//
// The activation row is staged once per CTA in fp32 (a decode step keeps all its activations in
// fp32, so the only 16-bit operand is the stored weight) and, where the layer's norm is one
// number, the norm is one factor per row that the epilogue applies.  A CTA owns a contiguous
// range of rows; its eight warps form eight / KS row groups of KS warps that split the columns,
// four rows at a time per group, so that every activation value read from shared memory feeds
// four weights and each lane has eight 16-byte weight loads in flight.  Partial sums meet in
// shared memory once per CTA and are added in warp order.
#include <algorithm>

#include "dense.h"

namespace smelt {

namespace {

constexpr int kThreads = 256, kWarps = 8, kRowsPerPass = 4, kChunkCols = 256;

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

template <int MODE>
__global__ void __launch_bounds__(kThreads, 3) dense_matvec_kernel(const DenseMatvecArgs a, int rows_per_cta, int ks) {
    extern __shared__ __align__(16) float smem[];
    const int chunks = (a.cols + kChunkCols - 1) / kChunkCols;
    float* sx = smem;                          // [chunks][2][32][4]: a lane's eight values as two conflict-free halves
    float* part = smem + (size_t)chunks * kChunkCols;
    __shared__ float s_sum[kWarps];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int kid = warp % ks, group = warp / ks, groups = kWarps / ks;
    const int r0 = blockIdx.x * rows_per_cta, r1 = min(a.rows, r0 + rows_per_cta);
    pdl_trigger();

    // the first weights do not depend on the launch in front
    uint4 first[kRowsPerPass];
    const int c_first = kid * kChunkCols + lane * 8, base_first = r0 + group * kRowsPerPass;
#pragma unroll
    for (int r = 0; r < kRowsPerPass; ++r)
        first[r] = (base_first + r < r1 && c_first < a.cols) ? ld_stream(reinterpret_cast<const uint4*>(a.w + (size_t)(base_first + r) * a.cols + c_first)) : make_uint4(0, 0, 0, 0);

    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    float ss = 0.f;
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

    for (int base = base_first; base < r1; base += groups * kRowsPerPass) {
        float acc[kRowsPerPass] = {0.f, 0.f, 0.f, 0.f};
        const bf16* w0 = a.w + (size_t)base * a.cols + lane * 8;
        const int left = r1 - base;
#pragma unroll 2
        for (int c = kid; c < chunks; c += ks) {
            const int col = c * kChunkCols + lane * 8;
            if (col < a.cols) {
                uint4 wv[kRowsPerPass];
#pragma unroll
                for (int r = 0; r < kRowsPerPass; ++r)
                    wv[r] = base == base_first && c == kid ? first[r]
                            : r < left                     ? ld_stream(reinterpret_cast<const uint4*>(w0 + (size_t)r * a.cols + c * kChunkCols))
                                                           : make_uint4(0, 0, 0, 0);
                const float4 xa = *reinterpret_cast<const float4*>(sx + c * kChunkCols + lane * 4);
                const float4 xb = *reinterpret_cast<const float4*>(sx + c * kChunkCols + 128 + lane * 4);
#pragma unroll
                for (int r = 0; r < kRowsPerPass; ++r) acc[r] = dot8(wv[r], xa, xb, acc[r]);
            }
        }
#pragma unroll
        for (int r = 0; r < kRowsPerPass; ++r) acc[r] = warp_sum(acc[r]);
        if (lane < kRowsPerPass && lane < left) part[(size_t)(base - r0 + lane) * ks + kid] = lane == 0 ? acc[0] : lane == 1 ? acc[1] : lane == 2 ? acc[2] : acc[3];
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
    const size_t x_bytes = (size_t)chunks * kChunkCols * sizeof(float), limit = 220 * 1024;
    // as many CTAs as are resident at once, each with an equal share of the rows (at least one pass of its row groups)
    int resident = (int)(limit / (x_bytes + 8192));
    resident = resident < 1 ? 1 : resident > 3 ? 3 : resident;
    int rows_per_cta = (a.rows + resident * sm - 1) / (resident * sm);
    rows_per_cta = std::max(rows_per_cta, std::min(kRowsPerPass * (kWarps / ks), 8));
    const int grid = (a.rows + rows_per_cta - 1) / rows_per_cta;
    const size_t smem = x_bytes + (size_t)rows_per_cta * ks * sizeof(float);
    if (smem > limit) return cudaErrorInvalidValue;
    return mode == kDenseAddF32 ? launch_chained(l, dense_matvec_kernel<kDenseAddF32>, dim3(grid), dim3(kThreads), smem, a, rows_per_cta, ks)
                                : launch_chained(l, dense_matvec_kernel<kDenseStoreF32>, dim3(grid), dim3(kThreads), smem, a, rows_per_cta, ks);
}

}  // namespace smelt
