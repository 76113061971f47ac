// The weight stream of the matrix-vector kernels of a decoded token (dense_matvec.cu,
// stack_matvec.cu): bf16 weights straight from global memory against an fp32 activation row in
// shared memory.
//
// A CTA owns a contiguous range of rows; its sixteen warps form 16 / ks row groups of ks warps that
// split the columns.  A warp's work is a sequence of items of four rows x 256 columns, so that every
// activation value read from shared memory feeds four weights; kDepth items are in flight in
// registers (256 bytes a lane), across the end of a group of rows and, where the weights do not
// depend on it, across the wait for the launch in front.  Partial sums go to shared memory, [row of
// the CTA][ks], and are added in warp order by the caller.
#pragma once
#include "dense.h"

namespace smelt {
namespace matvec {

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

// Column i (a multiple of 4) of the activation row in shared memory: a lane's eight values as two conflict-free halves.
__device__ __forceinline__ int staged(int i) {
    const int in = i % kChunkCols;
    return i - in + ((in >> 2) & 1) * 128 + (in >> 3) * 4;
}

// ks and the rows a CTA takes: one CTA per SM with an equal share, at least what keeps its row groups busy.
struct Split {
    int chunks, ks, rows_per_cta;
    size_t smem() const { return (size_t)chunks * kChunkCols * sizeof(float) + (size_t)rows_per_cta * ks * sizeof(float); }
};
inline Split split_rows(int rows, int cols, int sm_count) {
    const int sm = sm_count > 0 ? sm_count : 148;
    Split s;
    s.chunks = (cols + kChunkCols - 1) / kChunkCols;
    s.ks = 1;
    while (s.ks < kWarps && s.ks * 2 <= s.chunks) s.ks *= 2;
    const int least = kRowsPerPass * (kWarps / s.ks);
    s.rows_per_cta = (rows + sm - 1) / sm;
    if (s.rows_per_cta < (least < 8 ? least : 8)) s.rows_per_cta = least < 8 ? least : 8;
    return s;
}
constexpr size_t kMaxShared = 225 * 1024;

// Rows [r0, r1) of one CTA: their products with the staged activation row sx go to part, [r1 - r0][ks].
// Rows: first(row, col) is where a lane's eight columns of a row lie, after(first, r) the same of the r-th row behind it.
// prepare() waits for the launch in front and stages the activations (ending in a barrier), false: nothing
// is to be done; the first weights are requested ahead of it, or behind it where they depend on it (!EARLY).
template <bool EARLY, class Rows, class Prepare>
__device__ __forceinline__ bool stream_rows(const Rows& rows, int r0, int r1, int cols, int chunks, int ks, const float* sx, float* part, Prepare prepare) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kid = warp % ks, group = warp / ks, step = kWarps / ks * kRowsPerPass;
    struct Item { int row, chunk; };
    auto next = [&](Item& it) {
        it.chunk += ks;
        if (it.chunk >= chunks) { it.chunk = kid; it.row += step; }
    };
    auto load = [&](const Item& it, uint4 (&dst)[kRowsPerPass]) {
        const int col = it.chunk * kChunkCols + lane * 8;
        const auto p = rows.first(it.row, col);
        const bool in = col < cols;
#pragma unroll
        for (int r = 0; r < kRowsPerPass; ++r) dst[r] = in && it.row + r < r1 ? ld_stream(rows.after(p, r)) : make_uint4(0, 0, 0, 0);
    };
    uint4 buf[kDepth][kRowsPerPass];
    Item cur{r0 + group * kRowsPerPass, kid}, ahead = cur;
    if (EARLY) {
#pragma unroll
        for (int i = 0; i < kDepth; ++i) { load(ahead, buf[i]); next(ahead); }
    }
    pdl_trigger();  // behind the first requests: ahead of them it cost 0.9 us
    if (!prepare()) return false;
    if (!EARLY) {
#pragma unroll
        for (int i = 0; i < kDepth; ++i) { load(ahead, buf[i]); next(ahead); }
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
    return true;
}

// Rows of one matrix.
struct MatrixRows {
    const bf16* w;
    int cols;
    __device__ __forceinline__ const uint4* first(int row, int col) const { return reinterpret_cast<const uint4*>(w + (size_t)row * cols + col); }
    __device__ __forceinline__ const uint4* after(const uint4* p, int r) const { return p + (size_t)r * (cols / 8); }
};

__device__ __forceinline__ float sum_parts(const float* part, int i, int ks) {
    float v = 0.f;
    for (int k = 0; k < ks; ++k) v += part[(size_t)i * ks + k];
    return v;
}

// The sum of v over the CTA's threads, the same in all of them (one barrier; scratch: kWarps floats used once).
__device__ __forceinline__ float cta_sum(float v, float* scratch) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) tot += scratch[w];
    return tot;
}

}  // namespace matvec
}  // namespace smelt
