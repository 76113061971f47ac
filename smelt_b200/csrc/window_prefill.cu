// Window + pooled-block attention of a prompt chunk on the tensor cores.
//
// The query heads that share a KV head are rows beside their positions: row = position * ratio +
// head, 64 consecutive rows per CTA whatever the ratio, 16 per warp.  The CTA walks the blocks its
// last position sees and then the window from its first position's start, 64 keys at a time; K and
// V tiles are copied with cp.async into one of two swizzled buffers while the other is used.
// S = Q K^T and O = P V with mma.sync m16n8k16 (bf16, fp32 accumulate), P as the sum of two bf16
// values.  Weights need no running maximum (window.cuh), so nothing is rescaled.  Only tiles that
// some row does not see in full are masked.
#include "attention.cuh"
#include "window.cuh"

namespace smelt {

namespace {

constexpr int kRows = 64, kKeys = 64, kThreads = 128;

__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

// Byte offset of 16-byte piece c of row r in a tile of rows of N elements: pieces of eight
// neighbouring rows fall into different banks.
template <int N> __device__ __forceinline__ uint32_t piece(int r, int c) { return (uint32_t)(r * (N * 2) + ((c ^ (r & 7)) << 4)); }

template <int D, int VD> __host__ __device__ constexpr size_t prefill_smem() { return (size_t)kRows * D * 2 + 2 * (size_t)kKeys * (D + VD) * 2; }

template <int D, int VD>
__global__ void __launch_bounds__(kThreads) window_prefill_kernel(const WindowArgs a, const CapWeight cw) {
    constexpr bool kQInRegs = D <= 128;
    constexpr int KS = D / 16;  // k steps of a score
    extern __shared__ __align__(128) unsigned char smem[];
    unsigned char* sQ = smem;
    unsigned char* sK = sQ + kRows * D * 2;          // [2]
    unsigned char* sV = sK + 2 * kKeys * D * 2;      // [2]
    pdl_trigger();
    pdl_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int kvh = blockIdx.y, ratio = a.heads / a.kv_heads, total = a.m * ratio;
    const int row0 = blockIdx.x * kRows, row_last = min(total, row0 + kRows) - 1;
    const uint32_t start = dyn_position(a.dyn), first = start + row0 / ratio, last = start + row_last / ratio;
    const uint32_t nb_last = min(visible_blocks(last, a.window, a.pool), a.blocks), nb_first = min(visible_blocks(first, a.window, a.pool), a.blocks);
    const uint32_t lo = window_start(first, a.window), lo_last = window_start(last, a.window), lo_slot = lo % a.ring;
    const int pool_tiles = (int)((nb_last + kKeys - 1) / kKeys), tiles = pool_tiles + (int)((last + 1u - lo + kKeys - 1) / kKeys);
    const size_t head_rows = a.ring + a.blocks;
    const bf16* K = static_cast<const bf16*>(a.k_cache) + kvh * head_rows * D;
    const bf16* V = static_cast<const bf16*>(a.v_cache) + kvh * head_rows * VD;

    auto issue_tile = [&](int tile, int buf) {
        auto copy = [&](int r, int c, int n, unsigned char* dst, const bf16* base, uint32_t off) {
            uint32_t row;
            if (tile < pool_tiles) row = a.ring + min((uint32_t)(tile * kKeys + r), nb_last - 1u);
            else {
                row = lo_slot + min((uint32_t)((tile - pool_tiles) * kKeys + r), last - lo);
                if (row >= a.ring) row -= a.ring;
            }
            cp_async16(dst + off, base + (size_t)row * n + c * 8);
        };
        for (int i = tid; i < kKeys * (D / 8); i += kThreads) { const int r = i / (D / 8), c = i % (D / 8); copy(r, c, D, sK + buf * kKeys * D * 2, K, piece<D>(r, c)); }
        for (int i = tid; i < kKeys * (VD / 8); i += kThreads) { const int r = i / (VD / 8), c = i % (VD / 8); copy(r, c, VD, sV + buf * kKeys * VD * 2, V, piece<VD>(r, c)); }
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

    // this thread's two rows: lane / 4 and lane / 4 + 8 of the warp's sixteen
    const int my0 = min(row0 + warp * 16 + (lane >> 2), row_last), my1 = min(row0 + warp * 16 + (lane >> 2) + 8, row_last);
    const uint32_t i0 = start + my0 / ratio, i1 = start + my1 / ratio;
    const uint32_t nb0 = min(visible_blocks(i0, a.window, a.pool), a.blocks), nb1 = min(visible_blocks(i1, a.window, a.pool), a.blocks);
    const uint32_t lo0 = window_start(i0, a.window), lo1 = window_start(i1, a.window);

    const uint32_t q_addr = smem_u32(sQ), q_row = warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, q_half = lane >> 4;
    uint32_t qf[kQInRegs ? KS : 1][4];
    float o[VD / 8][4], l0 = 0.f, l1 = 0.f;
#pragma unroll
    for (int n = 0; n < VD / 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;

    for (int tile = 0; tile < tiles; ++tile) {
        const int buf = tile & 1;
        if (tile + 1 < tiles) issue_tile(tile + 1, buf ^ 1);
        else cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        if (kQInRegs && tile == 0) {
#pragma unroll
            for (int k = 0; k < KS; ++k) ldsm_x4(qf[k], q_addr + piece<D>(q_row, 2 * k + q_half));
        }
        const uint32_t k_addr = smem_u32(sK + buf * kKeys * D * 2), v_addr = smem_u32(sV + buf * kKeys * VD * 2);
        const bool pooled = tile < pool_tiles;
        const uint32_t base = pooled ? (uint32_t)tile * kKeys : lo + (uint32_t)(tile - pool_tiles) * kKeys;  // block or position of the tile's first key
        const bool seen_in_full = pooled ? base + kKeys <= nb_first : base >= lo_last && base + kKeys - 1u <= first;

        float s[kKeys / 8][4];
#pragma unroll
        for (int n = 0; n < kKeys / 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
#pragma unroll
        for (int k = 0; k < KS; ++k) {
            uint32_t qr[4];
            if (!kQInRegs) ldsm_x4(qr, q_addr + piece<D>(q_row, 2 * k + q_half));
            const uint32_t(&qv)[4] = kQInRegs ? qf[kQInRegs ? k : 0] : qr;
#pragma unroll
            for (int n = 0; n < kKeys / 16; ++n) {
                uint32_t kf[4];
                ldsm_x4(kf, k_addr + piece<D>(n * 16 + (lane & 7) + (lane >> 4) * 8, 2 * k + ((lane >> 3) & 1)));
                mma16816_bf16(s[2 * n], qv[0], qv[1], qv[2], qv[3], kf[0], kf[1]);
                mma16816_bf16(s[2 * n + 1], qv[0], qv[1], qv[2], qv[3], kf[2], kf[3]);
            }
        }
#pragma unroll
        for (int n = 0; n < kKeys / 8; ++n)
#pragma unroll
            for (int c = 0; c < 4; ++c) s[n][c] = cap_weight_of(cw, s[n][c]);
        if (!seen_in_full) {
#pragma unroll
            for (int n = 0; n < kKeys / 8; ++n)
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    const uint32_t key = base + n * 8 + 2 * (lane & 3) + (c & 1);
                    const bool seen = pooled ? key < (c < 2 ? nb0 : nb1) : key >= (c < 2 ? lo0 : lo1) && key <= (c < 2 ? i0 : i1);
                    if (!seen) s[n][c] = 0.f;
                }
        }
#pragma unroll
        for (int n = 0; n < kKeys / 8; ++n) { l0 += s[n][0] + s[n][1]; l1 += s[n][2] + s[n][3]; }
#pragma unroll
        for (int k = 0; k < kKeys / 16; ++k) {
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
                ldsm_x4_trans(vf, v_addr + piece<VD>(k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, 2 * n + (lane >> 4)));
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
    const float f0 = 1.f / (l0 + cw.sink), f1 = 1.f / (l1 + cw.sink);
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int row = row0 + warp * 16 + (lane >> 2) + half * 8;
        if (row >= total) continue;
        const float f = half ? f1 : f0;
        bf16* z = static_cast<bf16*>(a.z) + (size_t)(row / ratio) * a.ldz + (kvh * ratio + row % ratio) * a.vdim;
#pragma unroll
        for (int n = 0; n < VD / 8; ++n) {
            const int d = n * 8 + 2 * (lane & 3);
            const float x = o[n][2 * half] * f, y = o[n][2 * half + 1] * f;
            if (a.vdim % 2 == 0) {
                if (d < a.vdim) *reinterpret_cast<uint32_t*>(z + d) = attn::TileElem<bf16>::pack(x, y);
            } else {
                if (d < a.vdim) z[d] = from_f32<bf16>(x);
                if (d + 1 < a.vdim) z[d + 1] = from_f32<bf16>(y);
            }
        }
    }
}

template <int D, int VD>
cudaError_t launch_t(const Launch& l, const WindowArgs& a) {
    const dim3 grid((unsigned)(((size_t)a.m * (a.heads / a.kv_heads) + kRows - 1) / kRows), a.kv_heads);
    return launch_chained(l, window_prefill_kernel<D, VD>, grid, dim3(kThreads), prefill_smem<D, VD>(), a, cap_weight(a.scale, a.softcap));
}

template <int D>
cudaError_t launch_values(const Launch& l, const WindowArgs& a) {
    switch (a.vp) {
        case 64: return launch_t<D, 64>(l, a);
        case 128: return launch_t<D, 128>(l, a);
        default: return launch_t<D, 256>(l, a);
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
