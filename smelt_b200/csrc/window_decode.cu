// One decode step of the window + pooled-block attention in one launch: query and key norm, cache
// append, attention, merge of the key ranges, block mean.
//
// Grid (splits, KV heads x groups of up to 16 query heads); the splits of a head cut its visible
// keys (blocks first, then the window in position order) into equal ranges and form a
// thread-block cluster.  Eight warps walk 16-key tiles with the flash-decode tile functions
// (attention.cuh): keys on the MMA's M, query heads on its N, each lane's operands copied with
// cp.async into its own slots of a ring, so no barrier stands between a copy and its use.  Rows
// written by earlier tokens are requested before the wait for the launch in front; the tile with
// the new token's row is requested after the CTA that owns it has written the row.  Weights need
// no running maximum (window.cuh), so warps and ranks merge by addition: each rank pushes its sums
// into the shared memory of the rank that finishes a slice of the output.
#include <utility>

#include "attention.cuh"
#include "window.cuh"

namespace smelt {

namespace {

using namespace attn;

template <int D, int VD> __host__ __device__ constexpr int unit_bytes() { return (D > VD ? D : VD) / 16 * 512; }
template <int D, int VD> __host__ __device__ constexpr int ring_units_of() { return D > 128 || VD > 128 ? 2 : 3; }
// Bytes: the rings and the normed queries; over them, once the keys are done, the warps' sums; then what other ranks push.
template <int D, int VD, int NH> __host__ __device__ constexpr size_t recv_offset() {
    const size_t loop = (size_t)kAttnWarps * ring_units_of<D, VD>() * unit_bytes<D, VD>() + (size_t)NH * 8 * D * 2;
    const size_t merge = (size_t)kAttnWarps * NH * 8 * (VD + 1) * sizeof(float);
    return ((loop > merge ? loop : merge) + 15) & ~(size_t)15;
}
template <int D, int VD, int NH> __host__ __device__ constexpr size_t decode_smem() {
    return recv_offset<D, VD, NH>() + ((size_t)NH * 8 * VD + 8 + 8 * NH * 8) * sizeof(float);
}

template <int D, int VD, int NH>
__global__ void __launch_bounds__(kAttnThreads) window_decode_kernel(const WindowArgs a, const CapWeight cw, int head_groups) {
    constexpr int NU = ring_units_of<D, VD>(), UB = unit_bytes<D, VD>(), KJ = D / 32, VC = VD / 64, HN = NH * 8;
    extern __shared__ __align__(16) unsigned char smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int splits = gridDim.x, split = blockIdx.x, kvh = blockIdx.y / head_groups, hgroup = blockIdx.y % head_groups;
    const int ratio = a.heads / a.kv_heads, head0 = kvh * ratio + hgroup * HN, heads = min(HN, ratio - hgroup * HN);

    // The position was set before this token's first launch.
    const uint32_t i = dyn_position(a.dyn);
    const uint32_t nb = min(visible_blocks(i, a.window, a.pool), a.blocks), lo = window_start(i, a.window), n = nb + (i + 1u - lo);
    const uint32_t first_slot = lo % a.ring;
    uint32_t per = (n + splits - 1) / splits;
    per = (per + 15u) & ~15u;
    const uint32_t k_begin = min(n, (uint32_t)split * per), k_end = min(n, k_begin + per);
    const bool owner = k_begin < n && k_end == n;  // of the new token's key, the last one
    const size_t head_rows = a.ring + a.blocks;
    bf16* K = static_cast<bf16*>(a.k_cache) + kvh * head_rows * D;
    bf16* V = static_cast<bf16*>(a.v_cache) + kvh * head_rows * VD;
    auto cache_row = [&](uint32_t key) {
        if (key < nb) return a.ring + key;
        const uint32_t s = first_slot + (key - nb);
        return s >= a.ring ? s - a.ring : s;
    };

    unsigned char* ring = smem + (size_t)warp * NU * UB + lane * 16;
    const uint32_t kt0 = k_begin + warp * 16;
    auto issue_unit = [&](int u) {  // K (even) or V (odd) of this warp's tile u / 2
        const uint32_t kt = kt0 + (uint32_t)(u >> 1) * (kAttnWarps * 16);
        if (kt < k_end) {
            unsigned char* dst = ring + (size_t)(u % NU) * UB;
            const uint32_t last = k_end - 1;  // rows past the end repeat the last key, their weights are zero
            if ((u & 1) == 0) {
                const bf16* ka = K + (size_t)cache_row(min(kt + g, last)) * D + 8 * t;
                const bf16* kb = K + (size_t)cache_row(min(kt + g + 8, last)) * D + 8 * t;
#pragma unroll
                for (int j = 0; j < KJ; ++j) {
                    cp_async16(dst + (2 * j) * 512, ka + 32 * j);
                    cp_async16(dst + (2 * j + 1) * 512, kb + 32 * j);
                }
            } else {
#pragma unroll
                for (int kk = 0; kk < 4; ++kk) {
                    const bf16* v = V + (size_t)cache_row(min(kt + 2 * t + (kk & 1) + 8 * (kk >> 1), last)) * VD + 8 * g;
#pragma unroll
                    for (int c = 0; c < VC; ++c) cp_async16(dst + (4 * c + kk) * 512, v + 64 * c);
                }
            }
        }
        cp_async_commit();  // always: the group count stays uniform past the last tile
    };
    int issued = 0;
    for (; issued < NU - 1; ++issued) {
        const uint32_t kt = kt0 + (uint32_t)(issued >> 1) * (kAttnWarps * 16);
        if (kt < k_end && kt + 16 > n - 1u) break;  // holds the new token's row
        issue_unit(issued);
    }
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) {
        cp_async_wait<0>();
        return;
    }
    cg::cluster_group cluster = cg::this_cluster();
    auto started = cluster.barrier_arrive();  // nobody pushes into a rank that has not begun

    // ── norms and append: one warp per query head, then the new key and value ──
    bf16* sq = reinterpret_cast<bf16*>(smem + (size_t)kAttnWarps * NU * UB);
    const float* u = static_cast<const float*>(a.u);
    const uint32_t slot = i % a.ring;
    for (int item = warp; item < heads + (owner ? 2 : 0); item += kAttnWarps) {
        if (item == heads + 1) {
            const float* src = u + (a.heads + a.kv_heads) * a.dim + kvh * a.vdim;
            for (int d = lane; d < a.vdim; d += 32) V[(size_t)slot * VD + d] = from_f32<bf16>(src[d]);
            continue;
        }
        const float* src = u + (item < heads ? head0 + item : a.heads + kvh) * a.dim;
        const bf16* w = item < heads ? a.q_norm : a.k_norm;
        float v[D / 32], ss = 0.f;
#pragma unroll
        for (int j = 0; j < D / 32; ++j) {
            const int d = lane + 32 * j;
            v[j] = d < a.dim ? src[d] : 0.f;
            ss = fmaf(v[j], v[j], ss);
        }
        const float f = rsqrtf(warp_sum(ss) / (float)a.dim + a.eps);
        bf16* dst = item < heads ? sq + item * D : K + (size_t)slot * D;
#pragma unroll
        for (int j = 0; j < D / 32; ++j) {
            const int d = lane + 32 * j;
            dst[d] = from_f32<bf16>(d < a.dim ? v[j] * f * to_f32(w[d]) : 0.f);
        }
    }
    __threadfence_block();
    __syncthreads();

    uint32_t qf[NH][D / 8];
#pragma unroll
    for (int nh = 0; nh < NH; ++nh)
#pragma unroll
        for (int j = 0; j < KJ; ++j) {
            const int h = nh * 8 + g;
            const uint4 v = h < heads ? *reinterpret_cast<const uint4*>(sq + h * D + 32 * j + 8 * t) : make_uint4(0, 0, 0, 0);
            qf[nh][4 * j + 0] = v.x; qf[nh][4 * j + 1] = v.y; qf[nh][4 * j + 2] = v.z; qf[nh][4 * j + 3] = v.w;
        }
    for (; issued < NU - 1; ++issued) issue_unit(issued);

    float l_run[NH][2], o[NH][VD / 16][4];
#pragma unroll
    for (int nh = 0; nh < NH; ++nh) {
        l_run[nh][0] = l_run[nh][1] = 0.f;
#pragma unroll
        for (int m = 0; m < VD / 16; ++m) o[nh][m][0] = o[nh][m][1] = o[nh][m][2] = o[nh][m][3] = 0.f;
    }
    int unit = 0;
    for (uint32_t kt = kt0; kt < k_end; kt += kAttnWarps * 16, unit += 2) {
        const bool va = kt + g < k_end, vb = kt + g + 8 < k_end;
        issue_unit(unit + NU - 1);
        cp_async_wait<NU - 1>();
        float s[NH][4];
        tile_scores<D, NH, bf16>(ring + (size_t)(unit % NU) * UB, qf, s);
        uint32_t pb0[NH], pb1[NH], pl0[NH], pl1[NH];
#pragma unroll
        for (int nh = 0; nh < NH; ++nh) {
            const float p0 = va ? cap_weight_of(cw, s[nh][0]) : 0.f, p1 = va ? cap_weight_of(cw, s[nh][1]) : 0.f;
            const float p2 = vb ? cap_weight_of(cw, s[nh][2]) : 0.f, p3 = vb ? cap_weight_of(cw, s[nh][3]) : 0.f;
            l_run[nh][0] += p0 + p2;
            l_run[nh][1] += p1 + p3;
            // a weight as the sum of two bf16 values
            const uint32_t pa = TileElem<bf16>::pack(p0, p1), pb = TileElem<bf16>::pack(p2, p3);
            const float2 fa = TileElem<bf16>::unpack(pa), fb = TileElem<bf16>::unpack(pb);
            pb0[nh] = movmatrix_trans(pa);
            pb1[nh] = movmatrix_trans(pb);
            pl0[nh] = movmatrix_trans(TileElem<bf16>::pack(p0 - fa.x, p1 - fa.y));
            pl1[nh] = movmatrix_trans(TileElem<bf16>::pack(p2 - fb.x, p3 - fb.y));
        }
        issue_unit(unit + NU);
        cp_async_wait<NU - 1>();
        tile_weighted_sum<VD, NH, bf16>(ring + (size_t)((unit + 1) % NU) * UB, o, pb0, pb1, pl0, pl1);
    }
#pragma unroll
    for (int nh = 0; nh < NH; ++nh)
#pragma unroll
        for (int off = 4; off < 32; off <<= 1) {
            l_run[nh][0] += __shfl_xor_sync(0xffffffffu, l_run[nh][0], off);
            l_run[nh][1] += __shfl_xor_sync(0xffffffffu, l_run[nh][1], off);
        }

    // ── add the warps' sums, in the rings' memory ──
    cp_async_wait<0>();
    __syncthreads();
    float* so = reinterpret_cast<float*>(smem);  // [warps][HN][VD]
    float* sl = so + kAttnWarps * HN * VD;       // [warps][HN]
#pragma unroll
    for (int nh = 0; nh < NH; ++nh) {
        if (g == 0) {
            sl[warp * HN + nh * 8 + 2 * t] = l_run[nh][0];
            sl[warp * HN + nh * 8 + 2 * t + 1] = l_run[nh][1];
        }
#pragma unroll
        for (int m = 0; m < VD / 16; ++m)
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const int j = 2 * m + (c >> 1), dim = 64 * (j >> 3) + 8 * g + (j & 7);
                so[(size_t)(warp * HN + nh * 8 + 2 * t + (c & 1)) * VD + dim] = o[nh][m][c];
            }
    }
    __syncthreads();
    float* recv = reinterpret_cast<float*>(smem + recv_offset<D, VD, NH>());  // [ranks][slice] sums of the outputs, then [ranks][HN] of the weights
    float* recv_l = recv + HN * VD + 8;
    cluster.barrier_wait(std::move(started));
    const int items = heads * VD, slice = (items + splits - 1) / splits;
    float* z = static_cast<float*>(a.z) + head0 * a.vdim;
    for (int idx = tid; idx < items; idx += kAttnThreads) {
        const int h = idx / VD, d = idx % VD;
        float acc = 0.f, l = 0.f;
#pragma unroll
        for (int w = 0; w < kAttnWarps; ++w) {
            acc += so[(size_t)(w * HN + h) * VD + d];
            l += sl[w * HN + h];
        }
        if (splits == 1) {
            if (d < a.vdim) z[h * a.vdim + d] = acc / (l + cw.sink);
            continue;
        }
        const int rank = idx / slice;
        cluster.map_shared_rank(recv, rank)[split * slice + (idx - rank * slice)] = acc;
        if (d == 0)
            for (int r = 0; r < splits; ++r) cluster.map_shared_rank(recv_l, r)[split * HN + h] = l;
    }
    if (splits > 1) {
        cluster.sync();
        for (int idx = split * slice + tid; idx < min(items, (split + 1) * slice); idx += kAttnThreads) {
            const int h = idx / VD, d = idx % VD;
            float acc = 0.f, l = 0.f;
            for (int r = 0; r < splits; ++r) {
                acc += recv[r * slice + (idx - split * slice)];
                l += recv_l[r * HN + h];
            }
            if (d < a.vdim) z[h * a.vdim + d] = acc / (l + cw.sink);
        }
    }

    // ── the block that the new token completes (first seen by a later token) ──
    if (owner && hgroup == 0 && (i + 1u) % a.pool == 0u) {
        const uint32_t b = (i + 1u) / a.pool - 1u;
        if (b < a.blocks)
            for (int d = tid; d < a.dim + a.vdim; d += kAttnThreads) {
                if (d < a.dim) K[(size_t)(a.ring + b) * D + d] = from_f32<bf16>(block_mean(K, b * a.pool, a.pool, a.ring, D, d));
                else V[(size_t)(a.ring + b) * VD + d - a.dim] = from_f32<bf16>(block_mean(V, b * a.pool, a.pool, a.ring, VD, d - a.dim));
            }
    }
}

template <int D, int VD, int NH>
cudaError_t launch_t(const Launch& l, const WindowArgs& a, int head_groups, int splits) {
    auto kern = window_decode_kernel<D, VD, NH>;
    const size_t smem = decode_smem<D, VD, NH>();
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(splits, a.kv_heads * head_groups);
    cfg.blockDim = dim3(kAttnThreads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = l.stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = splits;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = l.pdl ? 2 : 1;
    prefer_max_shared(kern);
    return cudaLaunchKernelEx(&cfg, kern, a, cap_weight(a.scale, a.softcap), head_groups);
}

template <int D, int VD>
cudaError_t launch_heads(const Launch& l, const WindowArgs& a) {
    const int ratio = a.heads / a.kv_heads, per_group = ratio > 8 ? 16 : 8, head_groups = (ratio + per_group - 1) / per_group;
    const int sm = a.sm_count > 0 ? a.sm_count : 148;
    // Eight key ranges wherever there are keys for them: the count follows the geometry, not the
    // position, and only falls where the heads alone fill the GPU.
    int splits = (uint64_t)a.window + a.blocks >= 128u ? 8 : 1;
    while (splits > 1 && splits * a.kv_heads * head_groups > 2 * sm) splits /= 2;
    return per_group == 16 ? launch_t<D, VD, 2>(l, a, head_groups, splits) : launch_t<D, VD, 1>(l, a, head_groups, splits);
}

template <int D>
cudaError_t launch_values(const Launch& l, const WindowArgs& a) {
    switch (a.vp) {
        case 64: return launch_heads<D, 64>(l, a);
        case 128: return launch_heads<D, 128>(l, a);
        default: return launch_heads<D, 256>(l, a);
    }
}

}  // namespace

cudaError_t launch_window_decode_tiled(const Launch& l, const WindowArgs& a) {
    switch (a.kp) {
        case 64: return launch_values<64>(l, a);
        case 128: return launch_values<128>(l, a);
        default: return launch_values<256>(l, a);
    }
}

}  // namespace smelt
