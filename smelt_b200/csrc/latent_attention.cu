// Latent window attention: what surrounds the scores, and a form of the scores for any size.
//
// A cache row is a latent c and one rotated key part shared by all heads; the unrotated keys and the
// values of a head are uk c and uv c.  A decode step never forms them: a head's query goes through
// uk^T (latent_query_kernel), scores and weighted sums are taken over the latents themselves, and
// the sum goes through uv (latent_values_kernel, which also merges the key ranges of the tensor-core
// decode kernel).  A prompt chunk in bf16 forms the keys and values of its window with one matrix
// product over the ring and attends to them (latent_prefill.cu).
//
// Norms, angles, scores, weights and sums are fp32 (the angle's product and reduction fp64).
#include <algorithm>

#include "latent.cuh"

namespace smelt {

namespace {

constexpr int kThreads = 256, kWarps = kThreads / 32;

// The row's latent, normed, and its key part, rotated, into the ring; one CTA.
template <class TC>
__device__ __forceinline__ void append_row(const LatentArgs& a, const float* u, uint32_t pos, float* scratch) {
    const uint32_t slot = pos % a.ring;
    const float* c = u + a.qp;
    float ss = 0.f;
    for (int i = threadIdx.x; i < a.rank; i += kThreads) ss = fmaf(c[i], c[i], ss);
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = ss;
    __syncthreads();
    float tot = 0.f;
    for (int w = 0; w < kWarps; ++w) tot += scratch[w];
    const float f = rsqrtf(tot / (float)a.rank + a.eps);
    TC* dst = static_cast<TC*>(a.c_ring) + (size_t)slot * a.kr;
    for (int i = threadIdx.x; i < a.rank; i += kThreads) dst[i] = from_f32<TC>(c[i] * f * to_f32(a.kv_norm[i]));
    const float* kp = c + a.rank;
    TC* rot = static_cast<TC*>(a.rot_ring) + (size_t)slot * a.rp;
    for (int i = threadIdx.x; i < a.rot; i += kThreads) rot[i] = from_f32<TC>(rotated(kp, i, a.rot_dims, a.freq, pos));
}

// One CTA per row: the query latent normed to cq, and (own) the row appended.
template <class TC>
__global__ void __launch_bounds__(kThreads) latent_append_kernel(const LatentArgs a) {
    __shared__ float scratch[2][kWarps];
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    const int r = blockIdx.x;
    const float* u = a.u + (size_t)r * a.ldu;
    float ss = 0.f;
    for (int i = threadIdx.x; i < a.qp; i += kThreads) ss = fmaf(u[i], u[i], ss);  // zero past the latent
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) scratch[0][threadIdx.x >> 5] = ss;
    __syncthreads();
    float tot = 0.f;
    for (int w = 0; w < kWarps; ++w) tot += scratch[0][w];
    const float f = rsqrtf(tot / (float)a.q_rank + a.eps);
    TC* cq = static_cast<TC*>(a.cq) + (size_t)r * a.qp;
    for (int i = threadIdx.x; i < a.qp; i += kThreads) cq[i] = from_f32<TC>(u[i] * f * to_f32(a.q_norm[i]));
    if (a.own) append_row<TC>(a, u, dyn_position(a.dyn) + (uint32_t)r, scratch[1]);
}

// qa[r][h] = [uk^T q | rotated part]; a CTA takes kQueryCols latent elements of one head: sixteen lanes of
// eight elements side by side, sixteen groups of them over the rows of uk, whose first rows are
// requested before the wait for the launch in front.  The last y of a decode step's grid appends instead.
constexpr int kQueryCols = 128, kQueryDepth = 8;

template <class TC, class TQ>
__global__ void __launch_bounds__(kThreads) latent_query_kernel(const LatentArgs a, int append) {
    extern __shared__ float sq[];  // [dp]
    __shared__ float scratch[kWarps];
    __shared__ __align__(16) float s_sum[16][kQueryCols + 4];
    const int tid = threadIdx.x, r = blockIdx.z, h = blockIdx.y, grp = tid >> 4, c = blockIdx.x * kQueryCols + (tid & 15) * 8;
    const bool mine = h < a.heads && c < a.kr;
    const bf16* w = a.kv + (size_t)h * a.dp * a.kr + c;
    uint4 buf[kQueryDepth];
#pragma unroll
    for (int j = 0; j < kQueryDepth; ++j) {
        const int d = grp + 16 * j;
        buf[j] = mine && d < a.dp ? *reinterpret_cast<const uint4*>(w + (size_t)d * a.kr) : make_uint4(0, 0, 0, 0);
    }
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    const uint32_t pos = dyn_position(a.dyn) + (uint32_t)r;
    if (append && h == a.heads) {
        if (blockIdx.x == 0) append_row<TC>(a, a.u, pos, scratch);
        return;
    }
    const TQ* q = static_cast<const TQ*>(a.q) + ((size_t)r * a.heads + h) * (a.dp + a.rp);
    float* qa = a.qa + ((size_t)r * a.heads + h) * (a.kr + a.rp);
    for (int i = tid; i < a.dp; i += kThreads) sq[i] = to_f32(q[i]);
    if (blockIdx.x == 0)
        for (int i = tid; i < a.rp; i += kThreads) qa[a.kr + i] = i < a.rot ? rotated(q + a.dp, i, a.rot_dims, a.freq, pos) : 0.f;
    __syncthreads();
    float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    auto add = [&](const uint4& v, float x) {
        const uint32_t p[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            acc[2 * j] = fmaf(__uint_as_float(p[j] << 16), x, acc[2 * j]);
            acc[2 * j + 1] = fmaf(__uint_as_float(p[j] & 0xFFFF0000u), x, acc[2 * j + 1]);
        }
    };
#pragma unroll
    for (int j = 0; j < kQueryDepth; ++j)
        if (grp + 16 * j < a.dp) add(buf[j], sq[grp + 16 * j]);
    if (mine)
        for (int d = grp + 16 * kQueryDepth; d < a.dp; d += 16) add(*reinterpret_cast<const uint4*>(w + (size_t)d * a.kr), sq[d]);
#pragma unroll
    for (int j = 0; j < 8; ++j) s_sum[grp][(tid & 15) * 8 + j] = acc[j];
    __syncthreads();
    if (tid < kQueryCols && blockIdx.x * kQueryCols + tid < a.kr) {
        float v = 0.f;
#pragma unroll
        for (int g = 0; g < 16; ++g) v += s_sum[g][tid];
        qa[blockIdx.x * kQueryCols + tid] = v;
    }
}

// One CTA per (row, head), any size: tiles of one key per thread for the scores, then one latent
// element per thread for the weighted sum.  One split, its sum already divided.
template <class TC>
__global__ void __launch_bounds__(kThreads) latent_scores_simple_kernel(const LatentArgs a) {
    extern __shared__ float smem[];
    float* sq = smem;                 // [kr + rp]
    float* acc = sq + a.kr + a.rp;    // [kr]
    float* sp = acc + a.kr;           // [kThreads]
    float* red = sp + kThreads;       // [kWarps]
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = blockIdx.x, h = blockIdx.y;
    const uint32_t i = dyn_position(a.dyn) + (uint32_t)row, lo = i + 1u > a.window ? i + 1u - a.window : 0u, total = i + 1u - lo;
    const TC* C = static_cast<const TC*>(a.c_ring);
    const TC* R = static_cast<const TC*>(a.rot_ring);
    const float* q = a.qa + ((size_t)row * a.heads + h) * (a.kr + a.rp);
    for (int d = tid; d < a.kr + a.rp; d += kThreads) sq[d] = q[d];
    for (int d = tid; d < a.kr; d += kThreads) acc[d] = 0.f;
    __syncthreads();
    float m = -INFINITY, den = 0.f;
    for (uint32_t t0 = 0; t0 < total; t0 += kThreads) {
        const uint32_t n = t0 + tid;
        float s = -INFINITY;
        if (n < total) {
            const size_t slot = (lo + n) % a.ring;
            const TC *c = C + slot * a.kr, *rt = R + slot * a.rp;
            float dot = 0.f;
            for (int d = 0; d < a.rank; ++d) dot = fmaf(sq[d], to_f32(c[d]), dot);
            for (int d = 0; d < a.rot; ++d) dot = fmaf(sq[a.kr + d], to_f32(rt[d]), dot);
            s = dot * a.scale;
        }
        const float wm = warp_max(s);
        if (lane == 0) red[warp] = wm;
        __syncthreads();
        float mn = m;
        for (int w = 0; w < kWarps; ++w) mn = fmaxf(mn, red[w]);
        const float p = n < total ? expf(s - mn) : 0.f, corr = expf(m - mn);
        const float ws = warp_sum(p);
        sp[tid] = p;
        __syncthreads();
        if (lane == 0) red[warp] = ws;
        __syncthreads();
        den *= corr;
        for (int w = 0; w < kWarps; ++w) den += red[w];
        m = mn;
        const uint32_t cnt = min((uint32_t)kThreads, total - t0);
        for (int d = tid; d < a.rank; d += kThreads) {
            float o = acc[d] * corr;
            uint32_t slot = (lo + t0) % a.ring;
            for (uint32_t j = 0; j < cnt; ++j) {
                o = fmaf(sp[j], to_f32(C[(size_t)slot * a.kr + d]), o);
                slot = slot + 1u == a.ring ? 0u : slot + 1u;
            }
            acc[d] = o;
        }
        __syncthreads();
    }
    float* out = a.part + ((size_t)row * a.heads + h) * a.kr;
    for (int d = tid; d < a.kr; d += kThreads) out[d] = acc[d] / den;
    if (tid == 0) a.part_ml[(size_t)row * a.heads + h] = make_float2(0.f, 1.f);
}

// z[r][h] = uv (merged latent sum): a CTA merges the head's splits into shared memory, then its warps
// take rows of uv, eight weights a lane; a warp's first rows are requested before the wait for the
// launch in front.
constexpr int kValueDepth = 8;  // 16-byte pieces a lane holds

template <class TZ>
__global__ void __launch_bounds__(kThreads) latent_values_kernel(const LatentArgs a, int rows_per_cta) {
    extern __shared__ __align__(16) float sc[];  // [kr], then the splits' weights, then [row groups][kr] sums
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, r = blockIdx.z, h = blockIdx.y;
    const int v0 = blockIdx.x * rows_per_cta, v1 = min(a.vp, v0 + rows_per_cta), pieces = (a.kr + 255) / 256;  // of a row
    const bf16* uv = a.kv + ((size_t)a.heads * a.dp + (size_t)h * a.vp) * a.kr;
    auto load = [&](int n) {  // the warp's n-th piece: its rows are v0 + warp, v0 + warp + 8, ...
        const int v = v0 + warp + n / pieces * kWarps, i = n % pieces * 256 + lane * 8;
        return v < v1 && i < a.kr ? *reinterpret_cast<const uint4*>(uv + (size_t)v * a.kr + i) : make_uint4(0, 0, 0, 0);
    };
    uint4 buf[kValueDepth];
#pragma unroll
    for (int n = 0; n < kValueDepth; ++n) buf[n] = load(n);
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    // the splits' weights: exp(maximum - overall maximum) over the overall sum
    const float2* ml = a.part_ml + (size_t)r * a.splits * a.heads + h;
    float* sw = sc + a.kr;
    if (warp == 0) {
        float m = -INFINITY, den = 0.f;
        for (int s = lane; s < a.splits; s += 32) {
            const float2 v = ml[(size_t)s * a.heads];
            if (v.y > 0.f) m = fmaxf(m, v.x);
        }
        m = warp_max(m);
        for (int s = lane; s < a.splits; s += 32) {
            const float2 v = ml[(size_t)s * a.heads];
            const float w = v.y > 0.f ? expf(v.x - m) : 0.f;
            den = fmaf(v.y, w, den);
            sw[s] = w;
        }
        den = warp_sum(den);
        for (int s = lane; s < a.splits; s += 32) sw[s] /= den;
    }
    __syncthreads();
    // groups of threads take four latent elements each and every groups-th split
    float* ss = sc + ((a.kr + a.splits + 3) & ~3);
    const int cols = a.kr / 4, groups = max(1, kThreads / cols);
    for (int x = tid; x < cols * groups; x += kThreads) {
        const int g = x / cols, i = x % cols * 4;
        const float* p = a.part + ((size_t)r * a.splits * a.heads + h) * a.kr + i;
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int s = g; s < a.splits; s += groups) {
            const float w = sw[s];
            if (w != 0.f) {  // a split without keys has written no sums
                const float4 v = *reinterpret_cast<const float4*>(p + (size_t)s * a.heads * a.kr);
                acc.x = fmaf(v.x, w, acc.x); acc.y = fmaf(v.y, w, acc.y); acc.z = fmaf(v.z, w, acc.z); acc.w = fmaf(v.w, w, acc.w);
            }
        }
        *reinterpret_cast<float4*>(ss + (size_t)g * a.kr + i) = acc;
    }
    __syncthreads();
    for (int i = tid; i < a.kr; i += kThreads) {
        float v = 0.f;
        for (int g = 0; g < groups; ++g) v += ss[(size_t)g * a.kr + i];
        sc[i] = v;
    }
    __syncthreads();
    TZ* z = static_cast<TZ*>(a.z) + (size_t)r * a.ldz + (size_t)h * a.vp;
    const int total = (v1 - v0 - warp + kWarps - 1) / kWarps * pieces;
    float acc = 0.f;
    for (int n0 = 0; n0 < total; n0 += kValueDepth) {
#pragma unroll
        for (int j = 0; j < kValueDepth; ++j) {
            const int n = n0 + j;
            if (n >= total) break;
            const int i = n % pieces * 256 + lane * 8;
            if (i < a.kr) {
                const float4 x0 = *reinterpret_cast<const float4*>(sc + i), x1 = *reinterpret_cast<const float4*>(sc + i + 4);
                const uint32_t q[4] = {buf[j].x, buf[j].y, buf[j].z, buf[j].w};
                const float x[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
#pragma unroll
                for (int k = 0; k < 4; ++k) acc = fmaf(__uint_as_float(q[k] & 0xFFFF0000u), x[2 * k + 1], fmaf(__uint_as_float(q[k] << 16), x[2 * k], acc));
            }
            if (n % pieces == pieces - 1) {
                acc = warp_sum(acc);
                if (lane == 0) z[v0 + warp + n / pieces * kWarps] = from_f32<TZ>(acc);
                acc = 0.f;
            }
            buf[j] = load(n + kValueDepth);
        }
    }
}

bool bad(const LatentArgs& a) {
    return a.heads <= 0 || a.dim <= 0 || a.rot <= 0 || a.vdim <= 0 || a.rank <= 0 || a.rot_dims < 0 || a.rot_dims > a.rot || a.rot_dims % 2 || a.dp < a.dim || a.dp % 16 || a.rp < a.rot ||
           a.rp % 16 || a.vp < a.vdim || a.vp % 64 || a.kr < a.rank || a.kr % 64 || a.qp % 64 || a.m <= 0 || a.ring == 0;
}
bool short_ring(const LatentArgs& a) { return a.window == 0 || (uint64_t)a.ring + 1 < (uint64_t)a.window + (uint32_t)a.m; }

}  // namespace

int latent_splits(const LatentArgs& a, DenseType type) {
    if (type == kDenseF32 || a.m != 1 || !a.q_f32 || !latent_decode_tiled(a)) return 1;
    const int sm = a.sm_count > 0 ? a.sm_count : 148, groups = (a.heads + 15) / 16;
    const int tiles = (int)std::min<uint64_t>(((uint64_t)a.window + kLatentTile - 1) / kLatentTile, 4096u);
    return std::max(1, std::min(tiles, std::min(64, sm / groups)));
}

cudaError_t launch_latent_append(const Launch& l, DenseType type, LatentArgs a) {
    if (bad(a) || !a.u || !a.cq || (a.own && a.ldu < a.qp + a.rank + a.rot) || a.ldu < a.qp) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    return type == kDenseF32 ? launch_chained(l, latent_append_kernel<float>, dim3(a.m), dim3(kThreads), 0, a) : launch_chained(l, latent_append_kernel<bf16>, dim3(a.m), dim3(kThreads), 0, a);
}

cudaError_t launch_latent_query(const Launch& l, DenseType type, LatentArgs a, bool append) {
    if (bad(a) || (append && (a.m != 1 || !a.u || a.ldu < a.qp + a.rank + a.rot))) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    const dim3 grid((a.kr + kQueryCols - 1) / kQueryCols, a.heads + (append ? 1 : 0), a.m), block(kThreads);
    const size_t smem = (size_t)a.dp * sizeof(float);
    if (type == kDenseF32) return launch_chained(l, latent_query_kernel<float, float>, grid, block, smem, a, (int)append);
    return a.q_f32 ? launch_chained(l, latent_query_kernel<bf16, float>, grid, block, smem, a, (int)append) : launch_chained(l, latent_query_kernel<bf16, bf16>, grid, block, smem, a, (int)append);
}

cudaError_t launch_latent_scores(const Launch& l, DenseType type, LatentArgs a) {
    if (bad(a) || short_ring(a) || a.splits != latent_splits(a, type)) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    if (type == kDenseBf16 && a.m == 1 && a.q_f32 && latent_decode_tiled(a)) return launch_latent_decode_tiled(l, a);
    const size_t smem = (size_t)(2 * a.kr + a.rp + kThreads + kWarps) * sizeof(float);
    const dim3 grid(a.m, a.heads), block(kThreads);
    return type == kDenseF32 ? launch_chained(l, latent_scores_simple_kernel<float>, grid, block, smem, a) : launch_chained(l, latent_scores_simple_kernel<bf16>, grid, block, smem, a);
}

cudaError_t launch_latent_values(const Launch& l, DenseType type, LatentArgs a) {
    if (bad(a) || a.ldz < a.heads * a.vp || a.splits != latent_splits(a, type)) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    const int sm = a.sm_count > 0 ? a.sm_count : 148;
    int per = a.vp;  // rows of uv a CTA takes: enough CTAs for the GPU
    while (per > kWarps && (long)a.heads * a.m * ((a.vp + per - 1) / per) < sm) per = std::max(kWarps, per / 2);
    const dim3 grid((a.vp + per - 1) / per, a.heads, a.m), block(kThreads);
    const int groups = std::max(1, kThreads / (a.kr / 4));
    const size_t smem = (size_t)(((a.kr + a.splits + 3) & ~3) + groups * a.kr) * sizeof(float);
    return type == kDenseF32 || a.q_f32 ? launch_chained(l, latent_values_kernel<float>, grid, block, smem, a, per) : launch_chained(l, latent_values_kernel<bf16>, grid, block, smem, a, per);
}

}  // namespace smelt
