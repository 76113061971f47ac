// Window + pooled-block attention of a prompt chunk on the tensor cores.
//
// The query heads that share a KV head are rows beside their positions: row = position * ratio +
// head, 16 RG consecutive rows per CTA whatever the ratio.  The CTA walks the blocks its last
// position sees and then the window from its first position's start, 64 keys at a time; K and V
// tiles are copied with cp.async into one of two swizzled buffers while the other is used.  Eight
// warps: RG groups of sixteen rows times 8 / RG parts of a tile's keys, so that two CTAs give an SM
// sixteen warps to hide each other's latencies; the parts' sums are added at the end.  RG is 4, or 2
// where that leaves SMs without a CTA (the kernel is bound by the latency of one CTA's walk).
// S = Q K^T and O = P V with mma.sync m16n8k16 (bf16, fp32 accumulate), P as the sum of two bf16
// values.  Weights need no running maximum (window.cuh), so nothing is rescaled.  Only tiles that
// some row does not see in full are masked.
#include <type_traits>

#include "attention.cuh"
#include "window.cuh"

namespace smelt {

namespace {

constexpr int kKeys = 64, kThreads = 256;

__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

// Byte offset of 16-byte piece c of row r in a tile of rows of N elements: pieces of eight
// neighbouring rows fall into different banks.
template <int N> __device__ __forceinline__ uint32_t piece(int r, int c) { return (uint32_t)(r * (N * 2) + ((c ^ (r & 7)) << 4)); }

template <int D, int VD, int RG> __host__ __device__ constexpr size_t prefill_smem() { return (size_t)16 * RG * D * 2 + 2 * (size_t)kKeys * (D + VD) * 2; }

template <int D, int VD, int RG>
__global__ void __launch_bounds__(kThreads, D <= 128 && VD <= 128 ? 2 : 1) window_prefill_kernel(const WindowArgs a, const CapWeight cw) {
    constexpr int KS = D / 16;  // k steps of a score
    constexpr int kRows = 16 * RG, kParts = 8 / RG, kPart = kKeys / kParts;
    extern __shared__ __align__(128) unsigned char smem[];
    unsigned char* sQ = smem;
    unsigned char* sK = sQ + kRows * D * 2;          // [2]
    unsigned char* sV = sK + 2 * kKeys * D * 2;      // [2]
    pdl_trigger();
    pdl_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, rw = warp % RG, kp = warp / RG;
    const int kvh = blockIdx.y, ratio = a.heads / a.kv_heads, total = a.m * ratio;
    const int row0 = blockIdx.x * kRows, row_last = min(total, row0 + kRows) - 1;
    const uint32_t start = dyn_position(a.dyn), first = start + row0 / ratio, last = start + row_last / ratio;
    const uint32_t nb_last = min(visible_blocks(last, a.window, a.pool), a.blocks), nb_first = min(visible_blocks(first, a.window, a.pool), a.blocks);
    const uint32_t lo = window_start(first, a.window), lo_last = window_start(last, a.window), lo_slot = lo % a.ring;
    const int pool_tiles = (int)((nb_last + kKeys - 1) / kKeys), tiles = pool_tiles + (int)((last + 1u - lo + kKeys - 1) / kKeys);
    const size_t head_rows = a.ring + a.blocks;
    const bf16* K = static_cast<const bf16*>(a.k_cache) + kvh * head_rows * D;
    const bf16* V = static_cast<const bf16*>(a.v_cache) + kvh * head_rows * VD;

    // a thread copies the same 16-byte column of every kThreads / (N / 8)-th row, a multiple of eight rows apart
    auto copy_rows = [&](auto width, unsigned char* dst, const bf16* base, uint32_t row_first, bool contiguous, auto row_of) {
        constexpr int N = decltype(width)::value, kStep = kThreads / (N / 8);
        const int r0 = tid / (N / 8), c = tid % (N / 8);
        dst += piece<N>(r0, c);
        if (contiguous) {
            const bf16* src = base + (size_t)(row_first + r0) * N + c * 8;
#pragma unroll
            for (int j = 0; j < kKeys / kStep; ++j) cp_async16(dst + j * kStep * N * 2, src + (size_t)j * kStep * N);
        } else {
#pragma unroll
            for (int j = 0; j < kKeys / kStep; ++j) cp_async16(dst + j * kStep * N * 2, base + (size_t)row_of(r0 + j * kStep) * N + c * 8);
        }
    };
    auto issue_tile = [&](int tile, int buf) {
        const bool pooled = tile < pool_tiles;
        const uint32_t off = (uint32_t)(pooled ? tile : tile - pool_tiles) * kKeys, count = pooled ? nb_last : last - lo + 1u;
        uint32_t row_first = pooled ? a.ring + off : lo_slot + off;
        if (!pooled && row_first >= a.ring) row_first -= a.ring;
        const bool contiguous = off + kKeys <= count && (pooled || row_first + kKeys <= a.ring);
        auto row_of = [&](int r) {  // keys past the end repeat the last one, their weights are zero
            const uint32_t key = min(off + (uint32_t)r, count - 1u);
            if (pooled) return a.ring + key;
            const uint32_t s = lo_slot + key;
            return s >= a.ring ? s - a.ring : s;
        };
        copy_rows(std::integral_constant<int, D>(), sK + buf * kKeys * D * 2, K, row_first, contiguous, row_of);
        copy_rows(std::integral_constant<int, VD>(), sV + buf * kKeys * VD * 2, V, row_first, contiguous, row_of);
        cp_async_commit();
    };
    {
        const bf16* q = static_cast<const bf16*>(a.q);
        for (int i = tid; i < kRows * (D / 8); i += kThreads) {
            const int r = i / (D / 8), c = i % (D / 8), row = min(row0 + r, row_last);
            cp_async16(sQ + piece<D>(r, c), q + ((size_t)(row / ratio) * a.heads + kvh * ratio + row % ratio) * D + c * 8);
        }
    }
    issue_tile(0, 0);  // one group with the queries

    // this thread's two rows: lane / 4 and lane / 4 + 8 of the group's sixteen
    const int my0 = min(row0 + rw * 16 + (lane >> 2), row_last), my1 = min(row0 + rw * 16 + (lane >> 2) + 8, row_last);
    const uint32_t i0 = start + my0 / ratio, i1 = start + my1 / ratio;

    const int l7 = lane & 7, b3 = (lane >> 3) & 1, b4 = lane >> 4;
    const uint32_t q_addr = smem_u32(sQ) + (rw * 16 + l7 + b3 * 8) * (D * 2);
    const uint32_t k_row = (kp * kPart + l7 + b4 * 8) * (D * 2), v_row = (kp * kPart + l7 + b3 * 8) * (VD * 2);
    float o[VD / 8][4], l0 = 0.f, l1 = 0.f;
#pragma unroll
    for (int n = 0; n < VD / 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;

    for (int tile = 0; tile < tiles; ++tile) {
        const int buf = tile & 1;
        if (tile + 1 < tiles) issue_tile(tile + 1, buf ^ 1);
        else cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const uint32_t k_addr = smem_u32(sK + buf * kKeys * D * 2) + k_row, v_addr = smem_u32(sV + buf * kKeys * VD * 2) + v_row;
        const bool pooled = tile < pool_tiles;
        const uint32_t base = (pooled ? (uint32_t)tile * kKeys : lo + (uint32_t)(tile - pool_tiles) * kKeys) + kp * kPart;  // block or position of this part's first key
        const bool seen_in_full = pooled ? base + kPart <= nb_first : base >= lo_last && base + kPart - 1u <= first;

        float s[kPart / 8][4];
#pragma unroll
        for (int n = 0; n < kPart / 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
#pragma unroll
        for (int k = 0; k < KS; ++k) {
            uint32_t qf[4];
            ldsm_x4(qf, q_addr + (((2 * k + b4) ^ l7) << 4));
#pragma unroll
            for (int n = 0; n < kPart / 16; ++n) {
                uint32_t kf[4];
                ldsm_x4(kf, k_addr + n * 16 * D * 2 + (((2 * k + b3) ^ l7) << 4));
                mma16816_bf16(s[2 * n], qf[0], qf[1], qf[2], qf[3], kf[0], kf[1]);
                mma16816_bf16(s[2 * n + 1], qf[0], qf[1], qf[2], qf[3], kf[2], kf[3]);
            }
        }
#pragma unroll
        for (int n = 0; n < kPart / 8; ++n)
#pragma unroll
            for (int c = 0; c < 4; ++c) s[n][c] = cap_weight_of(cw, s[n][c]);
        if (!seen_in_full) {
            const uint32_t end0 = pooled ? min(visible_blocks(i0, a.window, a.pool), a.blocks) : i0 + 1u, end1 = pooled ? min(visible_blocks(i1, a.window, a.pool), a.blocks) : i1 + 1u;
            const uint32_t from0 = pooled ? 0u : window_start(i0, a.window), from1 = pooled ? 0u : window_start(i1, a.window);
#pragma unroll
            for (int n = 0; n < kPart / 8; ++n)
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    const uint32_t key = base + n * 8 + 2 * (lane & 3) + (c & 1);
                    if (key < (c < 2 ? from0 : from1) || key >= (c < 2 ? end0 : end1)) s[n][c] = 0.f;
                }
        }
#pragma unroll
        for (int n = 0; n < kPart / 8; ++n) { l0 += s[n][0] + s[n][1]; l1 += s[n][2] + s[n][3]; }
#pragma unroll
        for (int k = 0; k < kPart / 16; ++k) {
            uint32_t hi[4], lo4[4];
#pragma unroll
            for (int x = 0; x < 4; ++x) {  // (rows 0-7 | 8-15) of keys 0-7, then of keys 8-15
                const float p0 = s[2 * k + (x >> 1)][2 * (x & 1)], p1 = s[2 * k + (x >> 1)][2 * (x & 1) + 1];
                hi[x] = attn::TileElem<bf16>::pack(p0, p1);
                const float2 f = attn::TileElem<bf16>::unpack(hi[x]);
                lo4[x] = attn::TileElem<bf16>::pack(p0 - f.x, p1 - f.y);
            }
#pragma unroll
            for (int n = 0; n < VD / 16; ++n) {
                uint32_t vf[4];
                ldsm_x4_trans(vf, v_addr + k * 16 * VD * 2 + (((2 * n + b4) ^ l7) << 4));
                mma16816_bf16(o[2 * n], hi[0], hi[1], hi[2], hi[3], vf[0], vf[1]);
                mma16816_bf16(o[2 * n + 1], hi[0], hi[1], hi[2], hi[3], vf[2], vf[3]);
                mma16816_bf16(o[2 * n], lo4[0], lo4[1], lo4[2], lo4[3], vf[0], vf[1]);
                mma16816_bf16(o[2 * n + 1], lo4[0], lo4[1], lo4[2], lo4[3], vf[2], vf[3]);
            }
        }
        __syncthreads();  // the buffer may be refilled
    }
    cp_async_wait<0>();
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    // the other parts' sums, in the tiles' memory
    static_assert((size_t)(kParts - 1) * RG * (VD / 8) * 512 <= 2 * (size_t)kKeys * (D + VD) * 2 && (size_t)(kParts - 1) * RG * 256 <= (size_t)kRows * D * 2, "the sums fit where the tiles were");
    float4* so = reinterpret_cast<float4*>(sK) + (size_t)rw * (VD / 8) * 32 + lane;
    float2* sl = reinterpret_cast<float2*>(sQ) + rw * 32 + lane;
    constexpr int kSo = RG * (VD / 8) * 32, kSl = RG * 32;  // per part
    if (kp > 0) {
#pragma unroll
        for (int n = 0; n < VD / 8; ++n) so[(kp - 1) * kSo + n * 32] = make_float4(o[n][0], o[n][1], o[n][2], o[n][3]);
        sl[(kp - 1) * kSl] = make_float2(l0, l1);
    }
    __syncthreads();
    if (kp > 0) return;
#pragma unroll
    for (int p = 0; p < kParts - 1; ++p) {
        l0 += sl[p * kSl].x;
        l1 += sl[p * kSl].y;
    }
    const float f0 = 1.f / (l0 + cw.sink), f1 = 1.f / (l1 + cw.sink);
    const int r0 = row0 + rw * 16 + (lane >> 2), r1 = r0 + 8;
    auto out_row = [&](int row) { return static_cast<bf16*>(a.z) + (size_t)(row / ratio) * a.ldz + (kvh * ratio + row % ratio) * a.vdim; };
    bf16 *z0 = out_row(min(r0, row_last)), *z1 = out_row(min(r1, row_last));
#pragma unroll
    for (int n = 0; n < VD / 8; ++n) {
        const int d = n * 8 + 2 * (lane & 3);
#pragma unroll
        for (int p = 0; p < kParts - 1; ++p) {
            const float4 other = so[p * kSo + n * 32];
            o[n][0] += other.x; o[n][1] += other.y; o[n][2] += other.z; o[n][3] += other.w;
        }
        const float v[4] = {o[n][0] * f0, o[n][1] * f0, o[n][2] * f1, o[n][3] * f1};
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            if ((half ? r1 : r0) >= total) continue;
            bf16* z = half ? z1 : z0;
            if (a.vdim % 2 == 0) {
                if (d < a.vdim) *reinterpret_cast<uint32_t*>(z + d) = attn::TileElem<bf16>::pack(v[2 * half], v[2 * half + 1]);
            } else {
                if (d < a.vdim) z[d] = from_f32<bf16>(v[2 * half]);
                if (d + 1 < a.vdim) z[d + 1] = from_f32<bf16>(v[2 * half + 1]);
            }
        }
    }
}

template <int D, int VD, int RG>
cudaError_t launch_t(const Launch& l, const WindowArgs& a) {
    const dim3 grid((unsigned)(((size_t)a.m * (a.heads / a.kv_heads) + 16 * RG - 1) / (16 * RG)), a.kv_heads);
    return launch_chained(l, window_prefill_kernel<D, VD, RG>, grid, dim3(kThreads), prefill_smem<D, VD, RG>(), a, cap_weight(a.scale, a.softcap));
}

template <int D, int VD>
cudaError_t launch_rows(const Launch& l, const WindowArgs& a) {
    if constexpr (D <= 128 && VD <= 128) {
        const size_t ctas = ((size_t)a.m * (a.heads / a.kv_heads) + 63) / 64 * a.kv_heads;
        if (ctas <= (size_t)(a.sm_count > 0 ? a.sm_count : 148)) return launch_t<D, VD, 2>(l, a);
    }
    return launch_t<D, VD, 4>(l, a);
}

template <int D>
cudaError_t launch_values(const Launch& l, const WindowArgs& a) {
    switch (a.vp) {
        case 64: return launch_rows<D, 64>(l, a);
        case 128: return launch_rows<D, 128>(l, a);
        default: return launch_rows<D, 256>(l, a);
    }
}

}  // namespace

cudaError_t launch_window_prefill_tiled(const Launch& l, const WindowArgs& a) {
    switch (a.kp) {
        case 64: return launch_values<64>(l, a);
        case 128: return launch_values<128>(l, a);
        default: return launch_values<256>(l, a);
    }
}

}  // namespace smelt
