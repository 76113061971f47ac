// Matrix products of a prompt chunk: Y[m, rows] = X[m, cols] . W[rows, cols]^T, bf16 weights.
//
// gemm_bf16_kernel (bf16 activations): tcgen05.  The weight rows are the MMA's M (128 per tile),
// the chunk's positions its N (16 .. 256 per tile), so a tile's output is transposed on the way out:
// tensor-memory lane r is weight row r, and a warp stores 32 adjacent rows of one position at a
// time.  Warp 0 brings both operands with TMA (64 columns = one 128-byte swizzled row per stage,
// rows past the matrix or the chunk read as zero); one lane of warp 1 issues the MMAs; warps 2-5
// read the accumulator of the previous tile meanwhile (two accumulators in tensor memory).  CTAs
// are persistent, one per SM; neighbouring units share their weight tile.  A matrix with few
// tiles splits its columns: every part leaves fp32 sums in scratch and the last one to finish
// adds them in split order.  Weight tiles of the first stages are requested before the wait for
// the launch in front.  With experts, a unit is a row tile of one expert's matrix and up to BN rows
// of the activations that chose it, both taken from a table that an earlier launch has written.
//
// Every wait is bounded: on expiry the CTA raises bit 11 of the device error word, its roles stop,
// copies and MMAs in flight are waited for (bounded too) and the tensor memory is freed.
//
// gemm_f32_kernel: fp32 activations and arithmetic on the CUDA cores (the fp32 table).
#include <cuda.h>

#include <algorithm>

#include "dense.h"
#include "tcgen05.cuh"

namespace smelt {

namespace {

// xIELU for a bf16 result, without a branch: the curve's two halves add, each zero on the other's
// side.  The exponential's error (a few 2^-24 absolute near zero) is far below the result's rounding.
__device__ __forceinline__ float xielu_bf16(float z, float rising, float falling) {
    const float pos = fmaxf(z, 0.f), neg = fminf(z, 0.f);
    return fmaf(0.5f, z, fmaf(rising * pos, pos, falling * (exp2_approx(neg * 1.4426950408889634f) - 1.f - neg)));
}

// ── tcgen05 ─────────────────────────────────────────────────────────────────
constexpr int kBlockRows = 128, kBlockCols = 64, kGemmThreads = 192, kEpilogueThreads = 128;
constexpr uint32_t kATile = kBlockRows * kBlockCols * 2;

__host__ __device__ constexpr int gemm_stages(int bn) { return bn == 256 ? 4 : bn == 128 ? 6 : 8; }
__host__ __device__ constexpr uint32_t gemm_stage_bytes(int bn) { return kATile + (uint32_t)bn * kBlockCols * 2; }
__host__ __device__ constexpr uint32_t gemm_smem(int bn) { return gemm_stages(bn) * gemm_stage_bytes(bn) + 1024; }

__device__ __forceinline__ void tma_load_2d(void* dst, const CUtensorMap* map, int x, int y, uint64_t* bar) {
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(smem_u32(dst)), "l"(map), "r"(x), "r"(y),
                 "r"(smem_u32(bar))
                 : "memory");
}

// Waits for a phase; gives up after about a second, or as soon as another role has.
__device__ __forceinline__ bool wait_alive(uint64_t* bar, uint32_t parity, volatile uint32_t* dead) {
    for (uint32_t i = 0; i < (1u << 20); ++i) {
        uint32_t ok;
        asm volatile(
            "{\n\t.reg .pred p;\n\t"
            "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2, %3;\n\t"
            "selp.u32 %0, 1, 0, p;\n\t}"
            : "=r"(ok)
            : "r"(smem_u32(bar)), "r"(parity), "r"(1000u)
            : "memory");
        if (ok) return true;
        if (*dead) return false;
    }
    *dead = 1u;
    return false;
}

struct GemmPlan {
    int row_tiles, token_tiles, ksplit, units;
};

struct Unit {
    int n0, m0, count;   // first output row, first position, positions
    int wy, xy;          // first rows of the operands
    int kb0, kb1, tile, part;
};

template <int ACT, int N>
__device__ __forceinline__ void activate(float (&v)[N], const DenseOut& o) {
#pragma unroll
    for (int j = 0; j < N; ++j) {
        if (ACT == kDenseRelu2) { const float z = fmaxf(v[j], 0.f); v[j] = z * z; }
        else if (ACT == kDenseTanh) v[j] = tanhf(v[j]);
        else if (ACT == kDenseDecay) v[j] = expf(-expf(v[j]));
        else v[j] = xielu_bf16(v[j], o.rising, o.falling);
    }
}

// ACT: what the rows past the split go through; kDenseStoreF32: kDenseDecay, or anything else for nothing.
template <int BN, int MODE, int ACT, bool EXPERTS>
__global__ void __launch_bounds__(kGemmThreads, 1) gemm_bf16_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_x, const DenseGemmArgs a,
                                                                    const GemmPlan plan) {
    constexpr int kStages = gemm_stages(BN);
    constexpr uint32_t kStageBytes = gemm_stage_bytes(BN), kTmemCols = 2 * BN < 32 ? 32 : 2 * BN;
    constexpr int kChunk = BN < 32 ? BN : 32;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    __shared__ uint64_t full[kStages], empty[kStages], acc_full[2], acc_empty[2];
    __shared__ uint32_t s_tmem, s_dead, s_ticket, s_go;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int kblocks = a.cols / kBlockCols;

    pdl_trigger();
    if (tid == 0) {
        for (int i = 0; i < kStages; ++i) { mbar_init(&full[i], 1); mbar_init(&empty[i], 1); }
        for (int i = 0; i < 2; ++i) { mbar_init(&acc_full[i], 1); mbar_init(&acc_empty[i], kEpilogueThreads / 32); }
        s_dead = 0u;
        mbar_fence_init();
        fence_async_smem();
    }
    if (warp == 1) tmem_alloc(&s_tmem, kTmemCols);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s_tmem;
    volatile uint32_t* dead = &s_dead;

    int units = plan.units;
    if (EXPERTS) {
        pdl_wait();
        units = __ldcg(&a.table[0].x) * plan.row_tiles;
    }
    // the token tiles of a row tile are neighbours; with experts the row tiles of a table entry are
    auto unit_at = [&](int u) {
        Unit t;
        if (EXPERTS) {
            const int4 e = __ldcg(a.table + 1 + u / plan.row_tiles);
            t.n0 = u % plan.row_tiles * kBlockRows;
            t.m0 = t.xy = e.y;
            t.count = e.z;
            t.wy = e.x * a.rows + t.n0;
            t.kb0 = 0; t.kb1 = kblocks; t.tile = u; t.part = 0;
        } else {
            t.part = u % plan.ksplit;
            t.tile = u / plan.ksplit;
            t.n0 = t.wy = t.tile / plan.token_tiles * kBlockRows;
            t.m0 = t.xy = t.tile % plan.token_tiles * BN;
            if (a.group_rows) t.xy += min(t.n0 / a.group_rows, a.groups - 1) * a.x_group;
            t.count = min(BN, a.m - t.m0);
            t.kb0 = (int)((long)t.part * kblocks / plan.ksplit);
            t.kb1 = (int)((long)(t.part + 1) * kblocks / plan.ksplit);
        }
        return t;
    };

    if (warp == 0) {
        if (lane == 0) {
            uint32_t it = 0;  // stages issued so far
            // the first stages' weights, ahead of the dependency
            uint32_t early = 0;
            if (!EXPERTS) {
                if ((int)blockIdx.x < units) {
                    const Unit t = unit_at(blockIdx.x);
                    for (; early < kStages && (int)early < t.kb1 - t.kb0; ++early) {
                        mbar_arrive_expect_tx(&full[early], kStageBytes);
                        tma_load_2d(smem + early * kStageBytes, &map_w, (t.kb0 + (int)early) * kBlockCols, t.wy, &full[early]);
                    }
                }
                pdl_wait();
            }
            bool alive = true;
            for (int u = blockIdx.x; u < units && alive; u += gridDim.x) {
                const Unit t = unit_at(u);
                for (int kb = t.kb0; kb < t.kb1; ++kb, ++it) {
                    const uint32_t s = it % kStages, use = it / kStages;
                    uint8_t* dst = smem + s * kStageBytes;
                    if (it >= early) {
                        if (use > 0 && !(alive = wait_alive(&empty[s], (use - 1) & 1, dead))) break;
                        mbar_arrive_expect_tx(&full[s], kStageBytes);
                        tma_load_2d(dst, &map_w, kb * kBlockCols, t.wy, &full[s]);
                    }
                    tma_load_2d(dst + kATile, &map_x, kb * kBlockCols, t.xy, &full[s]);
                }
            }
            // no copy may land after the CTA has left
            for (uint32_t i = it > kStages ? it - kStages : 0; i < it; ++i) mbar_poll_bounded(&full[i % kStages], (i / kStages) & 1);
        }
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(kBlockRows >> 4) << 24);  // f32 += bf16 x bf16, K-major both
            uint32_t it = 0, done = 0;
            bool alive = true;
            for (int u = blockIdx.x; u < units && alive; u += gridDim.x, ++done) {
                const Unit t = unit_at(u);
                const uint32_t buf = done & 1, use = done >> 1;
                if (use > 0 && !(alive = wait_alive(&acc_empty[buf], (use - 1) & 1, dead))) break;
                tc_fence_after();
                for (int kb = t.kb0; kb < t.kb1; ++kb, ++it) {
                    const uint32_t s = it % kStages;
                    if (!(alive = wait_alive(&full[s], (it / kStages) & 1, dead))) break;
                    tc_fence_after();
                    const uint32_t w = smem_u32(smem + s * kStageBytes), x = w + kATile;
#pragma unroll
                    for (int k = 0; k < kBlockCols / 16; ++k)
                        umma_f16(tmem + buf * BN, smem_desc_sw128(w + k * 32), smem_desc_sw128(x + k * 32), idesc, (kb != t.kb0 || k != 0) ? 1u : 0u);
                    umma_commit(&empty[s]);
                }
                if (alive) umma_commit(&acc_full[buf]);
            }
            // MMAs in flight read shared memory and write tensor memory: wait for the last stage they were given
            if (it > 0) mbar_poll_bounded(&empty[(it - 1) % kStages], ((it - 1) / kStages) & 1);
        }
    } else {
        if (!EXPERTS) pdl_wait();
        const int quad = warp & 3, et = tid - 64;
        const uint32_t lane_base = tmem + ((uint32_t)(quad * 32) << 16);
        uint32_t done = 0;
        for (int u = blockIdx.x; u < units; u += gridDim.x, ++done) {
            const Unit t = unit_at(u);
            const int m0 = t.m0, tile = t.tile;
            const uint32_t buf = done & 1;
            bool alive = wait_alive(&acc_full[buf], (done >> 1) & 1, dead);
            if (plan.ksplit > 1) {  // the four warps meet below: they go on together or not at all
                if (!alive) *dead = 1u;
                asm volatile("bar.sync 1, %0;" ::"n"(kEpilogueThreads) : "memory");
                if (et == 0) s_go = *dead == 0u ? 1u : 0u;
                asm volatile("bar.sync 1, %0;" ::"n"(kEpilogueThreads) : "memory");
                alive = s_go != 0u;
            }
            if (!__all_sync(0xffffffffu, alive)) break;
            tc_fence_after();
            const int r = quad * 32 + lane, row = t.n0 + r, cnt = t.count;
            bool finish = true;
            if (plan.ksplit > 1) {
                float* mine = a.part_scratch + (size_t)u * (BN * kBlockRows);
                for (int c0 = 0; c0 < cnt; c0 += kChunk) {
                    uint32_t v[kChunk / 8][8];
#pragma unroll
                    for (int j = 0; j < kChunk / 8; ++j) tmem_ld8(lane_base + buf * BN + c0 + 8 * j, v[j]);
                    tmem_wait_ld();
#pragma unroll
                    for (int j = 0; j < kChunk; ++j) __stcg(mine + (size_t)(c0 + j) * kBlockRows + r, __uint_as_float(v[j / 8][j % 8]));
                }
                __threadfence();
                asm volatile("bar.sync 1, %0;" ::"n"(kEpilogueThreads) : "memory");
                if (et == 0) s_ticket = (uint32_t)atomicAdd(a.part_counters + tile, 1);
                asm volatile("bar.sync 1, %0;" ::"n"(kEpilogueThreads) : "memory");
                finish = s_ticket == (uint32_t)plan.ksplit - 1u;
                if (finish) {
                    __threadfence();
                    if (et == 0) a.part_counters[tile] = 0;
                }
            }
            if (finish) {
                const float* parts = a.part_scratch + (size_t)tile * plan.ksplit * (BN * kBlockRows) + r;
                for (int c0 = 0; c0 < cnt; c0 += kChunk) {  // positions, kChunk at a time: their loads are in flight together
                    float v[kChunk];
                    float old[MODE == kDenseAddF32 ? kChunk : 1];
                    if (MODE == kDenseAddF32 && row < a.rows) {  // in flight beside the sums
                        const float* y = static_cast<const float*>(a.out.y0) + (size_t)(m0 + c0) * a.out.ld0 + row;
#pragma unroll
                        for (int j = 0; j < kChunk; ++j)
                            if (MODE == kDenseAddF32) old[j] = c0 + j < cnt ? y[(size_t)j * a.out.ld0] : 0.f;
                    }
                    if (plan.ksplit > 1) {
#pragma unroll
                        for (int j = 0; j < kChunk; ++j) v[j] = __ldcg(parts + (size_t)(c0 + j) * kBlockRows);
                        for (int z = 1; z < plan.ksplit; ++z)
#pragma unroll
                            for (int j = 0; j < kChunk; ++j) v[j] += __ldcg(parts + (size_t)z * (BN * kBlockRows) + (size_t)(c0 + j) * kBlockRows);
                    } else {
                        uint32_t w[kChunk / 8][8];
#pragma unroll
                        for (int j = 0; j < kChunk / 8; ++j) tmem_ld8(lane_base + buf * BN + c0 + 8 * j, w[j]);
                        tmem_wait_ld();
#pragma unroll
                        for (int j = 0; j < kChunk; ++j) v[j] = __uint_as_float(w[j / 8][j % 8]);
                    }
                    if (MODE == kDenseStoreGlu) {
                        // lanes are (gate, up) pairs: the even one takes the even positions, the odd one the odd ones
                        const bool odd = lane & 1;
                        bf16* y = static_cast<bf16*>(a.out.y0) + (size_t)(m0 + c0) * a.out.ld0 + row / 2;
#pragma unroll
                        for (int j = 0; j < kChunk; j += 2) {
                            const float other = __shfl_xor_sync(0xffffffffu, odd ? v[j] : v[j + 1], 1);
                            const float z = clamped_glu(odd ? other : v[j], odd ? v[j + 1] : other, a.out.rising);
                            const int p = j + (odd ? 1 : 0);
                            if (row < a.rows && c0 + p < cnt) y[(size_t)p * a.out.ld0] = from_f32<bf16>(z);
                        }
                    } else if (row < a.rows) {
                        if (MODE != kDenseAddF32 && a.out.bias) {
                            const float b = to_f32(a.out.bias[row]);
#pragma unroll
                            for (int j = 0; j < kChunk; ++j) v[j] += b;
                        }
                        if (MODE == kDenseAddF32) {
                            float* y = static_cast<float*>(a.out.y0) + (size_t)(m0 + c0) * a.out.ld0 + row;
#pragma unroll
                            for (int j = 0; j < kChunk; ++j)
                                if (MODE == kDenseAddF32 && c0 + j < cnt) y[(size_t)j * a.out.ld0] = old[j] + v[j];
                        } else if (MODE == kDenseStoreF32 || (MODE == kDenseStoreMixed && row < a.out.split)) {
                            float* y = static_cast<float*>(a.out.y0) + (size_t)(m0 + c0) * a.out.ld0 + row;
                            if (MODE == kDenseStoreF32 && ACT == kDenseDecay) activate<ACT>(v, a.out);
#pragma unroll
                            for (int j = 0; j < kChunk; ++j)
                                if (c0 + j < cnt) y[(size_t)j * a.out.ld0] = v[j];
                        } else {
                            const bool act = MODE == kDenseStoreMixed || row >= a.out.split;
                            const int ld = act ? a.out.ld1 : a.out.ld0;
                            bf16* y = (act ? static_cast<bf16*>(a.out.y1) - a.out.split : static_cast<bf16*>(a.out.y0)) + (size_t)(m0 + c0) * ld + row;
                            if (act) activate<ACT>(v, a.out);
#pragma unroll
                            for (int j = 0; j < kChunk; ++j)
                                if (c0 + j < cnt) y[(size_t)j * ld] = from_f32<bf16>(v[j]);
                        }
                    }
                    __syncwarp();  // the next tensor-memory load needs the whole warp
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&acc_empty[buf]);
        }
    }
    if (tid == 0 && a.err && *dead) atomicOr(a.err, 0x800u);
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem, kTmemCols);
    }
}

using EncodeTiled = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                 CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

EncodeTiled encode_tiled() {
    static const EncodeTiled fn = [] {
        void* p = nullptr;
        cudaDriverEntryPointQueryResult found;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &found) != cudaSuccess || found != cudaDriverEntryPointSuccess) p = nullptr;
        return reinterpret_cast<EncodeTiled>(p);
    }();
    return fn;
}

// A row-major [rows, cols] bf16 matrix read in boxes of box_rows x 64 columns, 128-byte swizzle.
bool encode_rows(CUtensorMap* map, const void* base, int rows, int cols, int box_rows) {
    const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)cols * 2};
    const cuuint32_t box[2] = {kBlockCols, (cuuint32_t)box_rows}, step[2] = {1, 1};
    const EncodeTiled fn = encode_tiled();
    return fn && fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, step, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                    CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int BN>
cudaError_t launch_bf16_t(const Launch& l, int mode, const DenseGemmArgs& a, const GemmPlan& plan) {
    CUtensorMap mw, mx;
    const int groups = a.group_rows ? a.groups : 1;
    if (!encode_rows(&mw, a.w, a.table ? a.rows * a.experts : a.rows, a.cols, kBlockRows) || !encode_rows(&mx, a.x, a.m + (groups - 1) * a.x_group, a.cols, BN)) return cudaErrorInvalidValue;
    const dim3 grid(std::min(plan.units, a.sm_count > 0 ? a.sm_count : 148)), block(kGemmThreads);
    auto go = [&](auto kernel) { return launch_chained(l, kernel, grid, block, gemm_smem(BN), mw, mx, a, plan); };
    if (a.table) {
        if constexpr (BN >= 32 && BN <= 128) {
            if (mode == kDenseStoreF32) return go(gemm_bf16_kernel<BN, kDenseStoreF32, kDenseXielu, true>);
            if (mode == kDenseStoreGlu) return go(gemm_bf16_kernel<BN, kDenseStoreGlu, kDenseXielu, true>);
        }
        return cudaErrorInvalidValue;
    }
    switch (mode) {
        case kDenseStoreF32: return a.out.act == kDenseDecay ? go(gemm_bf16_kernel<BN, kDenseStoreF32, kDenseDecay, false>) : go(gemm_bf16_kernel<BN, kDenseStoreF32, kDenseXielu, false>);
        case kDenseAddF32: return go(gemm_bf16_kernel<BN, kDenseAddF32, kDenseXielu, false>);
        case kDenseStoreAct:
            switch (a.out.act) {
                case kDenseXielu: return go(gemm_bf16_kernel<BN, kDenseStoreAct, kDenseXielu, false>);
                case kDenseRelu2: return go(gemm_bf16_kernel<BN, kDenseStoreAct, kDenseRelu2, false>);
                case kDenseTanh: return go(gemm_bf16_kernel<BN, kDenseStoreAct, kDenseTanh, false>);
                default: return cudaErrorInvalidValue;
            }
        case kDenseStoreMixed:
            switch (a.out.act) {
                case kDenseRelu2: return go(gemm_bf16_kernel<BN, kDenseStoreMixed, kDenseRelu2, false>);
                case kDenseTanh: return go(gemm_bf16_kernel<BN, kDenseStoreMixed, kDenseTanh, false>);
                default: return cudaErrorInvalidValue;
            }
        default: return cudaErrorInvalidValue;
    }
}

// Tile width and column split with the shortest estimated time: waves of units, a unit being its
// column blocks at the slower of the tensor core (2 BN cycles a block) and the operand fill, plus
// its epilogue.
int plan_gemm(const DenseGemmArgs& a, GemmPlan* best) {
    const int sm = a.sm_count > 0 ? a.sm_count : 148, kblocks = a.cols / kBlockCols, row_tiles = (a.rows + kBlockRows - 1) / kBlockRows;
    double best_cost = 0;
    int best_bn = 0;
    for (int bn : {16, 32, 64, 128, 256}) {
        const int token_tiles = (a.m + bn - 1) / bn;
        if (token_tiles > 1 && bn < 64) continue;
        const long tiles = (long)row_tiles * token_tiles;
        for (int ks = 1; ks <= 16; ++ks) {
            if (ks > 1 && (tiles * ks > sm || ks * 4 > kblocks || tiles > 4096 || !a.part_scratch || !a.part_counters ||
                           (size_t)tiles * ks * bn * kBlockRows * sizeof(float) > a.part_scratch_bytes))
                break;
            const long units = tiles * ks, waves = (units + sm - 1) / sm;
            const double block = std::max(2.0 * bn, (double)gemm_stage_bytes(bn) / 64.0);
            const double cost = waves * ((kblocks + ks - 1) / ks) * block + 8.0 * bn + (ks > 1 ? 3000.0 + 4.0 * ks * bn : 0.0);
            if (best_bn == 0 || cost < best_cost) {
                best_cost = cost;
                best_bn = bn;
                *best = GemmPlan{row_tiles, token_tiles, ks, (int)units};
            }
        }
    }
    return best_bn;
}

cudaError_t launch_bf16(const Launch& l, int mode, const DenseGemmArgs& a) {
    GemmPlan plan;
    if (a.table) {
        const int row_tiles = (a.rows + kBlockRows - 1) / kBlockRows;
        plan = GemmPlan{row_tiles, 1, 1, row_tiles * a.max_entries};
        return a.tile == 32 ? launch_bf16_t<32>(l, mode, a, plan) : a.tile == 64 ? launch_bf16_t<64>(l, mode, a, plan) : a.tile == 128 ? launch_bf16_t<128>(l, mode, a, plan) : cudaErrorInvalidValue;
    }
    switch (plan_gemm(a, &plan)) {
        case 16: return launch_bf16_t<16>(l, mode, a, plan);
        case 32: return launch_bf16_t<32>(l, mode, a, plan);
        case 64: return launch_bf16_t<64>(l, mode, a, plan);
        case 128: return launch_bf16_t<128>(l, mode, a, plan);
        default: return launch_bf16_t<256>(l, mode, a, plan);
    }
}

// ── fp32 ────────────────────────────────────────────────────────────────────
constexpr int kTile = 64, kStep = 32;

template <int MODE>
__device__ __forceinline__ void store_f32(const DenseOut& o, int token, int row, float v) {
    if (o.bias) v += to_f32(o.bias[row]);
    float* y0 = static_cast<float*>(o.y0) + (size_t)token * o.ld0 + row;
    if (MODE == kDenseAddF32) { *y0 += v; return; }
    if (MODE == kDenseStoreF32) { *y0 = o.act == kDenseDecay ? expf(-expf(v)) : v; return; }
    if (row < o.split) { *y0 = v; return; }
    const float z = fmaxf(v, 0.f);
    static_cast<float*>(o.y1)[(size_t)token * o.ld1 + (row - o.split)] = o.act == kDenseRelu2 ? z * z : o.act == kDenseTanh ? tanhf(v) : xielu(v, o.rising, o.falling);
}

template <int MODE, bool EXPERTS>
__global__ void __launch_bounds__(256) gemm_f32_kernel(const DenseGemmArgs a, DevDyn dyn) {
    __shared__ float xs[kTile][kStep + 1], ws[kTile][kStep + 1];
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(dyn)) return;
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int n0 = blockIdx.x * kTile;
    int m0 = blockIdx.y * kTile, m1 = a.m;
    const bf16* w = a.w;
    const float* x = static_cast<const float*>(a.x);
    if (EXPERTS) {
        if ((int)blockIdx.y >= a.table[0].x) return;
        const int4 e = a.table[1 + blockIdx.y];
        m0 = e.y;
        m1 = e.y + e.z;
        w += (size_t)e.x * a.rows * a.cols;
    } else if (a.group_rows) {
        x += (size_t)min(n0 / a.group_rows, a.groups - 1) * a.x_group * a.cols;
    }
    float acc[4][4] = {};
    for (int k0 = 0; k0 < a.cols; k0 += kStep) {
        for (int i = tid; i < kTile * kStep; i += 256) {
            const int r = i / kStep, c = i % kStep;
            xs[r][c] = m0 + r < m1 ? x[(size_t)(m0 + r) * a.cols + k0 + c] : 0.f;
            ws[r][c] = n0 + r < a.rows ? to_f32(w[(size_t)(n0 + r) * a.cols + k0 + c]) : 0.f;
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
        for (int j = 0; j < 4; ++j) {
            const int token = m0 + ty + 16 * i, row = n0 + tx + 16 * j;
            if (MODE == kDenseStoreGlu) {  // the row beside it is the neighbouring thread's
                const float up = __shfl_xor_sync(0xffffffffu, acc[i][j], 1);
                if (token < m1 && row < a.rows && (tx & 1) == 0) static_cast<float*>(a.out.y0)[(size_t)token * a.out.ld0 + row / 2] = clamped_glu(acc[i][j], up, a.out.rising);
            } else if (token < m1 && row < a.rows) {
                store_f32<MODE>(a.out, token, row, acc[i][j]);
            }
        }
}

cudaError_t launch_f32(const Launch& l, int mode, const DenseGemmArgs& a) {
    const dim3 grid((a.rows + kTile - 1) / kTile, a.table ? a.max_entries : (a.m + kTile - 1) / kTile), block(256);
    if (a.table) {
        if (a.tile != kTile) return cudaErrorInvalidValue;
        if (mode == kDenseStoreF32) return launch_chained(l, gemm_f32_kernel<kDenseStoreF32, true>, grid, block, 0, a, dev_dyn(l));
        if (mode == kDenseStoreGlu) return launch_chained(l, gemm_f32_kernel<kDenseStoreGlu, true>, grid, block, 0, a, dev_dyn(l));
        return cudaErrorInvalidValue;
    }
    switch (mode) {
        case kDenseStoreF32: return launch_chained(l, gemm_f32_kernel<kDenseStoreF32, false>, grid, block, 0, a, dev_dyn(l));
        case kDenseAddF32: return launch_chained(l, gemm_f32_kernel<kDenseAddF32, false>, grid, block, 0, a, dev_dyn(l));
        case kDenseStoreAct: case kDenseStoreMixed: return launch_chained(l, gemm_f32_kernel<kDenseStoreAct, false>, grid, block, 0, a, dev_dyn(l));
        default: return cudaErrorInvalidValue;
    }
}

}  // namespace

cudaError_t launch_dense_gemm(const Launch& l, DenseType type, int mode, const DenseGemmArgs& a) {
    if (a.rows <= 0 || a.cols <= 0 || a.cols % 64 || a.m <= 0 || (mode != kDenseStoreAct && mode != kDenseStoreMixed && a.out.split != a.rows)) return cudaErrorInvalidValue;
    if ((a.group_rows && (a.group_rows % kBlockRows || a.x_group < a.m || a.groups <= 0)) || (a.table && (a.experts <= 0 || a.max_entries <= 0 || a.group_rows)) || (mode == kDenseStoreGlu && (!a.table || a.rows % kBlockRows)) || (mode == kDenseAddF32 && a.out.bias))
        return cudaErrorInvalidValue;
    if ((reinterpret_cast<uintptr_t>(a.w) | reinterpret_cast<uintptr_t>(a.x)) & 15u) return cudaErrorInvalidValue;
    return type == kDenseF32 ? launch_f32(l, mode, a) : launch_bf16(l, mode, a);
}

}  // namespace smelt
