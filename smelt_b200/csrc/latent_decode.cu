// Scores and weighted latent sums of one decoded token on the tensor cores (bf16 cache).
//
// All heads read the same rows, so sixteen heads are the MMA's M and the keys its N.  Grid (key
// ranges, groups of sixteen heads); a range is walked kLatentTile rows at a time, copied with
// cp.async into one of two buffers (rows of earlier tokens before the wait for the launch in
// front).  Scores: a warp takes eight keys and half of the row's elements; a query enters as the sum
// of two bf16 values.  Softmax with a running maximum: sixteen lanes a head.  Weighted sums: the same
// rows are the values, a warp takes an eighth of the latent's columns; weights are the sum of two
// bf16 values as well.  The ranges' sums stay unmerged: latent_values_kernel merges them.
#include "latent.cuh"

namespace smelt {

namespace {

constexpr int kThreads = 256, kHeads = 16, kKeys = kLatentTile, kMaxTiles = 8;  // 8-column tiles of a warp: kr <= 512

__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x2(uint32_t (&r)[2], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

// Bytes of a row of n elements in shared memory: rows start in different banks.
__host__ __device__ inline int pitch_of(int n) { return n * 2 + 16; }
constexpr int kPPitch = kKeys * 2 + 16;

__global__ void __launch_bounds__(kThreads) latent_decode_kernel(const LatentArgs a) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float s_part[2][kHeads][kKeys + 1];
    __shared__ __align__(16) unsigned char s_p[2][kHeads * kPPitch];  // weights: high and low halves
    __shared__ float s_corr[kHeads];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, split = blockIdx.x, head0 = blockIdx.y * kHeads;
    const int kd = a.kr + a.rp, pitch = pitch_of(kd), nt = a.kr / 64;
    unsigned char* sq = smem;                            // [2][kHeads] rows: high and low halves
    unsigned char* sk = smem + 2 * kHeads * pitch;       // [2][kKeys] rows
    const uint32_t i = dyn_position(a.dyn), lo = i + 1u > a.window ? i + 1u - a.window : 0u, n = i + 1u - lo;
    uint32_t per = (n + gridDim.x - 1) / gridDim.x;
    per = (per + kKeys - 1) / kKeys * kKeys;
    const uint32_t begin = min(n, (uint32_t)split * per), end = min(n, begin + per), lo_slot = lo % a.ring;
    const int tiles = (int)((end - begin + kKeys - 1) / kKeys);
    const bf16* C = static_cast<const bf16*>(a.c_ring);
    const bf16* R = static_cast<const bf16*>(a.rot_ring);
    auto copy_tile = [&](int tile, bool new_row, bool old_rows) {
        const uint32_t first = begin + (uint32_t)tile * kKeys;
        unsigned char* dst = sk + (tile & 1) * kKeys * pitch;
        const int pieces = kd / 8, c_pieces = a.kr / 8;
        for (int x = tid; x < kKeys * pieces; x += kThreads) {
            const int r = x / pieces, c = x % pieces;
            const uint32_t key = min(first + (uint32_t)r, end - 1u);  // rows past the end repeat the last key, their weights are zero
            if (key == n - 1u ? !new_row : !old_rows) continue;
            const uint32_t s = lo_slot + key, slot = s >= a.ring ? s - a.ring : s;
            cp_async16(dst + r * pitch + c * 16, c < c_pieces ? C + (size_t)slot * a.kr + c * 8 : R + (size_t)slot * a.rp + (c - c_pieces) * 8);
        }
    };
    if (tiles > 0) copy_tile(0, false, true);
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) {
        cp_async_commit();
        cp_async_wait<0>();
        return;
    }
    if (tiles == 0) {
        if (tid < kHeads && head0 + tid < a.heads) a.part_ml[(size_t)split * a.heads + head0 + tid] = make_float2(-INFINITY, 0.f);
        return;
    }
    copy_tile(0, true, false);
    cp_async_commit();
    for (int x = tid; x < kHeads * (kd / 2); x += kThreads) {
        const int h = x / (kd / 2), c = x % (kd / 2) * 2;
        float2 q = make_float2(0.f, 0.f);
        if (head0 + h < a.heads) q = *reinterpret_cast<const float2*>(a.qa + (size_t)(head0 + h) * kd + c);
        const __nv_bfloat162 hi = __floats2bfloat162_rn(q.x, q.y), lo2 = __floats2bfloat162_rn(q.x - __low2float(hi), q.y - __high2float(hi));
        *reinterpret_cast<__nv_bfloat162*>(sq + h * pitch + c * 2) = hi;
        *reinterpret_cast<__nv_bfloat162*>(sq + (kHeads + h) * pitch + c * 2) = lo2;
    }

    const int g = lane >> 2, t = lane & 3;
    const int ktile = warp & 3, khalf = warp >> 2, ksteps = kd / 16, k0 = khalf ? ksteps / 2 : 0, k1 = khalf ? ksteps : ksteps / 2;
    const uint32_t q_addr = smem_u32(sq) + (lane & 15) * pitch + (lane >> 4) * 16;
    const uint32_t k_off = (ktile * 8 + (lane & 7)) * pitch + ((lane >> 3) & 1) * 16;
    const int sh = tid >> 4, sj = tid & 15;  // softmax: head and first of the two keys (sj, sj + 16)
    float m_run = -INFINITY, l_run = 0.f;
    float o[kMaxTiles][4];
#pragma unroll
    for (int x = 0; x < kMaxTiles; ++x) o[x][0] = o[x][1] = o[x][2] = o[x][3] = 0.f;

    for (int tile = 0; tile < tiles; ++tile) {
        if (tile + 1 < tiles) copy_tile(tile + 1, true, true);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const uint32_t k_base = smem_u32(sk + (tile & 1) * kKeys * pitch);
        float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
        for (int k = k0; k < k1; ++k) {
            uint32_t qh[4], ql[4], kf[2];
            ldsm_x4(qh, q_addr + k * 32);
            ldsm_x4(ql, q_addr + kHeads * pitch + k * 32);
            ldsm_x2(kf, k_base + k_off + k * 32);
            mma16816_bf16(s, qh[0], qh[1], qh[2], qh[3], kf[0], kf[1]);
            mma16816_bf16(s2, ql[0], ql[1], ql[2], ql[3], kf[0], kf[1]);
        }
        s_part[khalf][g][ktile * 8 + 2 * t] = s[0] + s2[0];
        s_part[khalf][g][ktile * 8 + 2 * t + 1] = s[1] + s2[1];
        s_part[khalf][g + 8][ktile * 8 + 2 * t] = s[2] + s2[2];
        s_part[khalf][g + 8][ktile * 8 + 2 * t + 1] = s[3] + s2[3];
        __syncthreads();
        {
            const uint32_t first = begin + (uint32_t)tile * kKeys;
            float v[2];
#pragma unroll
            for (int x = 0; x < 2; ++x) v[x] = first + sj + 16 * x < end ? (s_part[0][sh][sj + 16 * x] + s_part[1][sh][sj + 16 * x]) * a.scale : -INFINITY;
            float mx = fmaxf(v[0], v[1]);
#pragma unroll
            for (int off = 8; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
            const float mn = fmaxf(m_run, mx), corr = expf(m_run - mn), p0 = expf(v[0] - mn), p1 = expf(v[1] - mn);
            float sum = p0 + p1;
#pragma unroll
            for (int off = 8; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
            l_run = fmaf(l_run, corr, sum);
            m_run = mn;
            if (sj == 0) s_corr[sh] = corr;
            const float p[2] = {p0, p1};
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const bf16 hi = from_f32<bf16>(p[x]);
                *reinterpret_cast<bf16*>(s_p[0] + sh * kPPitch + (sj + 16 * x) * 2) = hi;
                *reinterpret_cast<bf16*>(s_p[1] + sh * kPPitch + (sj + 16 * x) * 2) = from_f32<bf16>(p[x] - to_f32(hi));
            }
        }
        __syncthreads();
        uint32_t ph[2][4], pl[2][4];
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const uint32_t off = (lane & 15) * kPPitch + (lane >> 4) * 16 + k * 32;
            ldsm_x4(ph[k], smem_u32(s_p[0]) + off);
            ldsm_x4(pl[k], smem_u32(s_p[1]) + off);
        }
        const float c0 = s_corr[g], c1 = s_corr[g + 8];
#pragma unroll
        for (int x = 0; x < kMaxTiles; ++x) {
            if (x >= nt) break;
            uint32_t vf[4];  // 32 keys x 8 columns
            ldsm_x4_trans(vf, k_base + lane * pitch + (warp * nt + x) * 16);
            o[x][0] *= c0; o[x][1] *= c0; o[x][2] *= c1; o[x][3] *= c1;
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                mma16816_bf16(o[x], ph[k][0], ph[k][1], ph[k][2], ph[k][3], vf[2 * k], vf[2 * k + 1]);
                mma16816_bf16(o[x], pl[k][0], pl[k][1], pl[k][2], pl[k][3], vf[2 * k], vf[2 * k + 1]);
            }
        }
        __syncthreads();  // the buffers may be refilled
    }
    cp_async_wait<0>();
    float* part = a.part + ((size_t)split * a.heads + head0) * a.kr;
#pragma unroll
    for (int x = 0; x < kMaxTiles; ++x) {
        if (x >= nt) break;
        const int c = (warp * nt + x) * 8 + 2 * t;
        if (head0 + g < a.heads) *reinterpret_cast<float2*>(part + (size_t)g * a.kr + c) = make_float2(o[x][0], o[x][1]);
        if (head0 + g + 8 < a.heads) *reinterpret_cast<float2*>(part + (size_t)(g + 8) * a.kr + c) = make_float2(o[x][2], o[x][3]);
    }
    if (sj == 0 && head0 + sh < a.heads) a.part_ml[(size_t)split * a.heads + head0 + sh] = make_float2(m_run, l_run);
}

}  // namespace

cudaError_t launch_latent_decode_tiled(const Launch& l, const LatentArgs& a) {
    const size_t smem = (size_t)(2 * kHeads + 2 * kKeys) * pitch_of(a.kr + a.rp);
    return launch_chained(l, latent_decode_kernel, dim3(a.splits, (a.heads + kHeads - 1) / kHeads), dim3(kThreads), smem, a);
}

}  // namespace smelt
