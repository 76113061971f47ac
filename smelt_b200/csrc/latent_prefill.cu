// Latent window attention of a prompt chunk on the tensor cores, over keys and values that one
// product over the ring has formed (bf16).
//
// A CTA takes 16 RG consecutive positions of one head and walks the window of its last one from its
// first one's start, 64 keys at a time; a key's row in shared memory is its unrotated part and the
// rotated part that all heads share, its value stands beside it; both come with cp.async into one of
// two buffers while the other is used.  Queries are rotated on the way in.  Eight warps: RG groups of
// sixteen positions times 8 / RG parts of a tile's keys, each with its own running maximum; the
// parts merge at the end.  S = Q K^T and O = P V with mma.sync m16n8k16 (fp32 accumulate), P as the
// sum of two bf16 values.  RG is 4, or 2 where that leaves SMs without a CTA.
#include <type_traits>

#include "attention.cuh"
#include "latent.cuh"

namespace smelt {

namespace {

constexpr int kKeys = 64, kThreads = 256;

__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

// Bytes of a row of n elements (a multiple of 16) in shared memory: eight neighbouring rows fall into different banks.
__host__ __device__ constexpr int pitch_of(int n) { return n * 2 + 16; }
__host__ __device__ inline size_t merge_bytes(int vd, int rg) { return (size_t)(8 / rg - 1) * rg * 32 * (vd / 2 + 4) * sizeof(float); }
inline size_t prefill_smem(int d, int vd, int rg) {
    const size_t loop = (size_t)(16 * rg + 2 * kKeys) * pitch_of(d) + 2 * (size_t)kKeys * pitch_of(vd), merge = merge_bytes(vd, rg);
    return loop > merge ? loop : merge;
}

template <int VD, int RG>
__global__ void __launch_bounds__(kThreads, VD <= 128 ? 2 : 1) latent_prefill_kernel(const LatentArgs a) {
    constexpr int kRows = 16 * RG, kParts = 8 / RG, kPart = kKeys / kParts, kVPitch = pitch_of(VD);
    extern __shared__ __align__(16) unsigned char smem[];
    const int D = a.dp + a.rp, pitch = pitch_of(D), ksteps = D / 16;
    unsigned char* sQ = smem;
    unsigned char* sK = sQ + kRows * pitch;         // [2]
    unsigned char* sV = sK + 2 * kKeys * pitch;     // [2]
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, rw = warp % RG, kp = warp / RG, h = blockIdx.y;
    const int row0 = blockIdx.x * kRows, row_last = min(a.m, row0 + kRows) - 1;
    const uint32_t start = dyn_position(a.dyn), first = start + row0, last = start + row_last;
    auto window_start = [&](uint32_t i) { return i + 1u > a.window ? i + 1u - a.window : 0u; };
    const uint32_t lo = window_start(first), lo_last = window_start(last), lo_slot = lo % a.ring, count = last + 1u - lo;
    const int tiles = (int)((count + kKeys - 1) / kKeys);
    const int ld = a.heads * (a.dp + a.vp);
    const bf16* KV = static_cast<const bf16*>(a.kv_rows);
    const bf16* R = static_cast<const bf16*>(a.rot_ring);

    const int k_pieces = D / 8, d_pieces = a.dp / 8;
    auto issue_tile = [&](int tile, int buf) {
        auto slot_of = [&](int r) {  // keys past the end repeat the last one, their weights are zero
            const uint32_t s = lo_slot + min((uint32_t)(tile * kKeys + r), count - 1u);
            return s >= a.ring ? s - a.ring : s;
        };
        unsigned char *k = sK + buf * kKeys * pitch, *v = sV + buf * kKeys * kVPitch;
        // four threads a row
        const int r = tid >> 2, c0 = tid & 3;
        const uint32_t slot = slot_of(r);
        const bf16 *row = KV + (size_t)slot * ld, *rot = R + (size_t)slot * a.rp;
        for (int c = c0; c < k_pieces; c += 4) cp_async16(k + r * pitch + c * 16, c < d_pieces ? row + h * a.dp + c * 8 : rot + (c - d_pieces) * 8);
        const bf16* val = row + a.heads * a.dp + h * VD;
#pragma unroll
        for (int c = 0; c < VD / 32; ++c) cp_async16(v + r * kVPitch + (c0 + 4 * c) * 16, val + (c0 + 4 * c) * 8);
        cp_async_commit();
    };
    {
        const bf16* q = static_cast<const bf16*>(a.q) + (size_t)h * D;
        const int qld = a.heads * D;
        for (int x = tid; x < kRows * d_pieces; x += kThreads) {
            const int r = x / d_pieces, c = x % d_pieces;
            cp_async16(sQ + r * pitch + c * 16, q + (size_t)min(row0 + r, row_last) * qld + c * 8);
        }
        const int pairs = a.rp / 2;
        for (int x = tid; x < kRows * pairs; x += kThreads) {
            const int r = x / pairs, j = x % pairs, row = min(row0 + r, row_last);
            const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(q + (size_t)row * qld + a.dp + 2 * j);
            float2 w = make_float2(__low2float(v), __high2float(v));
            if (2 * j < a.rot_dims) {
                const float2 cs = rotary_cos_sin(start + row, a.freq[j]);
                w = make_float2(fmaf(w.x, cs.x, -w.y * cs.y), fmaf(w.y, cs.x, w.x * cs.y));
            }
            *reinterpret_cast<__nv_bfloat162*>(sQ + r * pitch + (a.dp + 2 * j) * 2) = __floats2bfloat162_rn(w.x, w.y);
        }
    }
    issue_tile(0, 0);  // one group with the queries

    // this thread's two rows: lane / 4 and lane / 4 + 8 of the group's sixteen
    const uint32_t i0 = start + min(row0 + rw * 16 + (lane >> 2), row_last), i1 = start + min(row0 + rw * 16 + (lane >> 2) + 8, row_last);
    const uint32_t from0 = window_start(i0), from1 = window_start(i1);
    const float rate = a.scale * 1.4426950408889634f;
    const int l7 = lane & 7, b3 = (lane >> 3) & 1, b4 = lane >> 4;
    const uint32_t q_addr = smem_u32(sQ) + (rw * 16 + l7 + b3 * 8) * pitch + b4 * 16;
    const uint32_t k_off = (kp * kPart + l7 + b4 * 8) * pitch + b3 * 16, v_off = (kp * kPart + l7 + b3 * 8) * kVPitch + b4 * 16;
    float o[VD / 8][4], l0 = 0.f, l1 = 0.f, m0 = -INFINITY, m1 = -INFINITY;
#pragma unroll
    for (int n = 0; n < VD / 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;

    for (int tile = 0; tile < tiles; ++tile) {
        const int buf = tile & 1;
        if (tile + 1 < tiles) issue_tile(tile + 1, buf ^ 1);
        else cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const uint32_t k_addr = smem_u32(sK + buf * kKeys * pitch) + k_off, v_addr = smem_u32(sV + buf * kKeys * kVPitch) + v_off;
        const uint32_t base = lo + (uint32_t)tile * kKeys + kp * kPart;  // position of this part's first key
        const bool seen_in_full = base >= lo_last && base + kPart - 1u <= first;
        if (base <= last) {
            float s[kPart / 8][4];
#pragma unroll
            for (int n = 0; n < kPart / 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
#pragma unroll 4
            for (int k = 0; k < ksteps; ++k) {
                uint32_t qf[4];
                ldsm_x4(qf, q_addr + k * 32);
#pragma unroll
                for (int n = 0; n < kPart / 16; ++n) {
                    uint32_t kf[4];
                    ldsm_x4(kf, k_addr + n * 16 * pitch + k * 32);
                    mma16816_bf16(s[2 * n], qf[0], qf[1], qf[2], qf[3], kf[0], kf[1]);
                    mma16816_bf16(s[2 * n + 1], qf[0], qf[1], qf[2], qf[3], kf[2], kf[3]);
                }
            }
            if (!seen_in_full) {
#pragma unroll
                for (int n = 0; n < kPart / 8; ++n)
#pragma unroll
                    for (int c = 0; c < 4; ++c) {
                        const uint32_t key = base + n * 8 + 2 * (lane & 3) + (c & 1);
                        if (key < (c < 2 ? from0 : from1) || key > (c < 2 ? i0 : i1)) s[n][c] = -INFINITY;
                    }
            }
            float x0 = -INFINITY, x1 = -INFINITY;
#pragma unroll
            for (int n = 0; n < kPart / 8; ++n) {
                x0 = fmaxf(x0, fmaxf(s[n][0], s[n][1]));
                x1 = fmaxf(x1, fmaxf(s[n][2], s[n][3]));
            }
            x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 1)); x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 2));
            x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 1)); x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 2));
            // maxima in units of log2; a row without a visible key yet keeps its sums at zero
            const float n0 = fmaxf(m0, x0 * rate), n1 = fmaxf(m1, x1 * rate);
            const float ref0 = n0 == -INFINITY ? 0.f : n0, ref1 = n1 == -INFINITY ? 0.f : n1;
            const float c0 = exp2_approx(m0 - ref0), c1 = exp2_approx(m1 - ref1);
            m0 = n0; m1 = n1;
            l0 *= c0; l1 *= c1;
#pragma unroll
            for (int n = 0; n < VD / 8; ++n) { o[n][0] *= c0; o[n][1] *= c0; o[n][2] *= c1; o[n][3] *= c1; }
#pragma unroll
            for (int n = 0; n < kPart / 8; ++n) {
                s[n][0] = exp2_approx(fmaf(s[n][0], rate, -ref0));
                s[n][1] = exp2_approx(fmaf(s[n][1], rate, -ref0));
                s[n][2] = exp2_approx(fmaf(s[n][2], rate, -ref1));
                s[n][3] = exp2_approx(fmaf(s[n][3], rate, -ref1));
                l0 += s[n][0] + s[n][1];
                l1 += s[n][2] + s[n][3];
            }
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
                    ldsm_x4_trans(vf, v_addr + k * 16 * kVPitch + n * 32);
                    mma16816_bf16(o[2 * n], hi[0], hi[1], hi[2], hi[3], vf[0], vf[1]);
                    mma16816_bf16(o[2 * n + 1], hi[0], hi[1], hi[2], hi[3], vf[2], vf[3]);
                    mma16816_bf16(o[2 * n], lo4[0], lo4[1], lo4[2], lo4[3], vf[0], vf[1]);
                    mma16816_bf16(o[2 * n + 1], lo4[0], lo4[1], lo4[2], lo4[3], vf[2], vf[3]);
                }
            }
        }
        __syncthreads();  // the buffer may be refilled
    }
    cp_async_wait<0>();
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    __syncthreads();
    // the other parts' sums and maxima, where the tiles were: [part][group][values][lane]
    float4* so = reinterpret_cast<float4*>(smem) + (size_t)rw * (VD / 8 + 1) * 32 + lane;
    constexpr int kSo = RG * (VD / 8 + 1) * 32;  // per part
    if (kp > 0) {
#pragma unroll
        for (int n = 0; n < VD / 8; ++n) so[(kp - 1) * kSo + n * 32] = make_float4(o[n][0], o[n][1], o[n][2], o[n][3]);
        so[(kp - 1) * kSo + VD / 8 * 32] = make_float4(m0, l0, m1, l1);
    }
    __syncthreads();
    if (kp > 0) return;
    float t0 = m0, t1 = m1, f0[kParts], f1[kParts];  // factors of the parts
#pragma unroll
    for (int p = 1; p < kParts; ++p) {
        const float4 v = so[(p - 1) * kSo + VD / 8 * 32];
        t0 = fmaxf(t0, v.x);
        t1 = fmaxf(t1, v.z);
    }
    f0[0] = exp2_approx(m0 - t0); f1[0] = exp2_approx(m1 - t1);
    float d0 = l0 * f0[0], d1 = l1 * f1[0];
#pragma unroll
    for (int p = 1; p < kParts; ++p) {
        const float4 v = so[(p - 1) * kSo + VD / 8 * 32];
        f0[p] = exp2_approx(v.x - t0); f1[p] = exp2_approx(v.z - t1);
        d0 = fmaf(v.y, f0[p], d0);
        d1 = fmaf(v.w, f1[p], d1);
    }
    d0 = 1.f / d0; d1 = 1.f / d1;
    const int r0 = row0 + rw * 16 + (lane >> 2), r1 = r0 + 8;
    bf16* z = static_cast<bf16*>(a.z) + (size_t)h * VD + 2 * (lane & 3);
#pragma unroll
    for (int n = 0; n < VD / 8; ++n) {
        float v[4] = {o[n][0] * f0[0], o[n][1] * f0[0], o[n][2] * f1[0], o[n][3] * f1[0]};
#pragma unroll
        for (int p = 1; p < kParts; ++p) {
            const float4 other = so[(p - 1) * kSo + n * 32];
            v[0] = fmaf(other.x, f0[p], v[0]); v[1] = fmaf(other.y, f0[p], v[1]);
            v[2] = fmaf(other.z, f1[p], v[2]); v[3] = fmaf(other.w, f1[p], v[3]);
        }
        if (r0 < a.m) *reinterpret_cast<uint32_t*>(z + (size_t)r0 * a.ldz + n * 8) = attn::TileElem<bf16>::pack(v[0] * d0, v[1] * d0);
        if (r1 < a.m) *reinterpret_cast<uint32_t*>(z + (size_t)r1 * a.ldz + n * 8) = attn::TileElem<bf16>::pack(v[2] * d1, v[3] * d1);
    }
}

template <int VD>
cudaError_t launch_rows(const Launch& l, const LatentArgs& a) {
    const int d = a.dp + a.rp, sm = a.sm_count > 0 ? a.sm_count : 148;
    if ((long)((a.m + 63) / 64) * a.heads <= sm)
        return launch_chained(l, latent_prefill_kernel<VD, 2>, dim3((a.m + 31) / 32, a.heads), dim3(kThreads), prefill_smem(d, VD, 2), a);
    return launch_chained(l, latent_prefill_kernel<VD, 4>, dim3((a.m + 63) / 64, a.heads), dim3(kThreads), prefill_smem(d, VD, 4), a);
}

}  // namespace

cudaError_t launch_latent_prefill(const Launch& l, LatentArgs a) {
    if (a.m <= 0 || a.window == 0 || (uint64_t)a.ring + 1 < (uint64_t)a.window + (uint32_t)a.m || !latent_prefill_tiled(a) || a.ldz < a.heads * a.vp) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    switch (a.vp) {
        case 64: return launch_rows<64>(l, a);
        case 128: return launch_rows<128>(l, a);
        case 256: return launch_rows<256>(l, a);
        default: return cudaErrorInvalidValue;
    }
}

}  // namespace smelt
