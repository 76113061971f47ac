// Attention over a sliding window and pooled blocks: head norms and cache append, block means,
// and the attention itself.
//
// Score s = (q . k) scale, then softcap tanh(s / softcap); the softmax has one more in its
// denominator (a sink with score 0 and no value).  Tokens of the window and pooled blocks share
// one softmax.  Norms, scores, weights and sums are fp32.
//
// The kernels here take any head size, softcap (or none) and cache type; with a bf16 cache, heads
// of up to 256 and a softcap the tensor-core kernels of window_decode.cu and window_prefill.cu run
// instead.
#include <algorithm>

#include "window.cuh"

namespace smelt {

namespace {

// One warp per head of a token: query heads normed to q, key heads normed into the ring, value
// heads copied into it.
template <class TC, class TU>
__global__ void __launch_bounds__(256) window_append_kernel(const WindowArgs a) {
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    const int lane = threadIdx.x & 31, item = blockIdx.y * 8 + (threadIdx.x >> 5), row = blockIdx.x;
    const int H = a.heads, G = a.kv_heads;
    if (item >= H + 2 * G) return;
    const TU* u = static_cast<const TU*>(a.u) + (size_t)row * (H * a.dim + G * (a.dim + a.vdim));
    const uint32_t slot = (dyn_position(a.dyn) + (uint32_t)row) % a.ring;
    const size_t head_rows = a.ring + a.blocks;
    if (item >= H + G) {
        const int g = item - H - G;
        const TU* src = u + (H + G) * a.dim + g * a.vdim;
        TC* dst = static_cast<TC*>(a.v_cache) + (g * head_rows + slot) * a.vp;
        for (int d = lane; d < a.vdim; d += 32) dst[d] = from_f32<TC>(to_f32(src[d]));
        return;
    }
    const TU* src = u + item * a.dim;
    const bf16* w = item < H ? a.q_norm : a.k_norm;
    float ss = 0.f;
    for (int d = lane; d < a.dim; d += 32) {
        const float v = to_f32(src[d]);
        ss = fmaf(v, v, ss);
    }
    const float f = rsqrtf(warp_sum(ss) / (float)a.dim + a.eps);
    if (item < H) {
        TU* dst = static_cast<TU*>(a.q) + ((size_t)row * H + item) * a.kp;
        for (int d = lane; d < a.kp; d += 32) dst[d] = from_f32<TU>(d < a.dim ? to_f32(src[d]) * f * to_f32(w[d]) : 0.f);
    } else {
        TC* dst = static_cast<TC*>(a.k_cache) + ((item - H) * head_rows + slot) * a.kp;
        for (int d = lane; d < a.dim; d += 32) dst[d] = from_f32<TC>(to_f32(src[d]) * f * to_f32(w[d]));
    }
}

template <class TC>
__global__ void __launch_bounds__(128) window_pool_kernel(const WindowArgs a) {
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    const uint32_t start = dyn_position(a.dyn), b = start / a.pool + blockIdx.x;
    if (b >= (start + (uint32_t)a.m) / a.pool || b >= a.blocks) return;
    const size_t head_rows = a.ring + a.blocks;
    TC* k = static_cast<TC*>(a.k_cache) + blockIdx.y * head_rows * a.kp;
    TC* v = static_cast<TC*>(a.v_cache) + blockIdx.y * head_rows * a.vp;
    for (int d = threadIdx.x; d < a.dim + a.vdim; d += blockDim.x) {
        if (d < a.dim) k[(size_t)(a.ring + b) * a.kp + d] = from_f32<TC>(block_mean(k, b * a.pool, a.pool, a.ring, a.kp, d));
        else v[(size_t)(a.ring + b) * a.vp + d - a.dim] = from_f32<TC>(block_mean(v, b * a.pool, a.pool, a.ring, a.vp, d - a.dim));
    }
}

// One CTA per (query row, head), any dim and vdim: tiles of one key per thread for the scores,
// then one value column per thread for the weighted sum.
constexpr int kSimpleThreads = 128;

template <class TC, class TU>
__global__ void __launch_bounds__(kSimpleThreads) window_attention_simple_kernel(const WindowArgs a) {
    extern __shared__ float smem[];
    float* sq = smem;           // [kp]
    float* acc = sq + a.kp;     // [vdim]
    float* sp = acc + a.vdim;   // [kSimpleThreads]
    float* red = sp + kSimpleThreads;
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = blockIdx.x, h = blockIdx.y, g = h / (a.heads / a.kv_heads);
    const uint32_t i = dyn_position(a.dyn) + (uint32_t)row;
    const uint32_t nb = min(visible_blocks(i, a.window, a.pool), a.blocks), lo = window_start(i, a.window), total = nb + (i + 1u - lo);
    const size_t head_rows = a.ring + a.blocks;
    const TC* K = static_cast<const TC*>(a.k_cache) + g * head_rows * a.kp;
    const TC* V = static_cast<const TC*>(a.v_cache) + g * head_rows * a.vp;
    const TU* q = static_cast<const TU*>(a.q) + ((size_t)row * a.heads + h) * a.kp;
    for (int d = tid; d < a.kp; d += kSimpleThreads) sq[d] = to_f32(q[d]);
    for (int d = tid; d < a.vdim; d += kSimpleThreads) acc[d] = 0.f;
    __syncthreads();
    auto cache_row = [&](uint32_t n) { return n < nb ? a.ring + n : (lo + (n - nb)) % a.ring; };
    float m = 0.f, den = 1.f;  // the sink: score 0, weight 1, no value
    for (uint32_t t0 = 0; t0 < total; t0 += kSimpleThreads) {
        const uint32_t n = t0 + tid;
        float s = -INFINITY;
        if (n < total) {
            const TC* k = K + (size_t)cache_row(n) * a.kp;
            float dot = 0.f;
            for (int d = 0; d < a.dim; ++d) dot = fmaf(sq[d], to_f32(k[d]), dot);
            s = dot * a.scale;
            if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
        }
        const float wm = warp_max(s);
        if (lane == 0) red[warp] = wm;
        __syncthreads();
        float mn = m;
        for (int w = 0; w < kSimpleThreads / 32; ++w) mn = fmaxf(mn, red[w]);
        const float p = n < total ? expf(s - mn) : 0.f, c = expf(m - mn);
        const float ws = warp_sum(p);
        sp[tid] = p;
        __syncthreads();
        if (lane == 0) red[warp] = ws;
        __syncthreads();
        den *= c;
        for (int w = 0; w < kSimpleThreads / 32; ++w) den += red[w];
        m = mn;
        const uint32_t cnt = min((uint32_t)kSimpleThreads, total - t0);
        for (int d = tid; d < a.vdim; d += kSimpleThreads) {
            float o = acc[d] * c;
            for (uint32_t j = 0; j < cnt; ++j) o = fmaf(sp[j], to_f32(V[(size_t)cache_row(t0 + j) * a.vp + d]), o);
            acc[d] = o;
        }
        __syncthreads();
    }
    TU* z = static_cast<TU*>(a.z) + (size_t)row * a.ldz + h * a.vdim;
    for (int d = tid; d < a.vdim; d += kSimpleThreads) z[d] = from_f32<TU>(acc[d] / den);
}

bool bad_geometry(const WindowArgs& a) {
    return a.heads <= 0 || a.kv_heads <= 0 || a.heads % a.kv_heads || a.dim <= 0 || a.vdim <= 0 || a.kp < a.dim || a.vp < a.vdim || a.window == 0 || a.pool == 0 || a.m <= 0 ||
           (uint64_t)a.ring + 1 < (uint64_t)std::max(a.window, a.pool) + (uint32_t)a.m;
}

template <class TC, class TU>
cudaError_t append_t(const Launch& l, const WindowArgs& a) {
    return launch_chained(l, window_append_kernel<TC, TU>, dim3(a.m, (a.heads + 2 * a.kv_heads + 7) / 8), dim3(256), 0, a);
}

template <class TC, class TU>
cudaError_t simple_t(const Launch& l, const WindowArgs& a) {
    const size_t smem = (size_t)(a.kp + a.vdim + kSimpleThreads + 32) * sizeof(float);
    return launch_chained(l, window_attention_simple_kernel<TC, TU>, dim3(a.m, a.heads), dim3(kSimpleThreads), smem, a);
}

}  // namespace

cudaError_t launch_window_append(const Launch& l, DenseType type, WindowArgs a) {
    if (bad_geometry(a)) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    if (type == kDenseF32) return append_t<float, float>(l, a);
    return a.u_f32 ? append_t<bf16, float>(l, a) : append_t<bf16, bf16>(l, a);
}

cudaError_t launch_window_pool(const Launch& l, DenseType type, WindowArgs a) {
    if (bad_geometry(a)) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    const dim3 grid((unsigned)a.m / a.pool + 1, a.kv_heads), block(128);
    return type == kDenseF32 ? launch_chained(l, window_pool_kernel<float>, grid, block, 0, a) : launch_chained(l, window_pool_kernel<bf16>, grid, block, 0, a);
}

cudaError_t launch_window_attention(const Launch& l, DenseType type, WindowArgs a) {
    if (bad_geometry(a)) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    if (type == kDenseF32) return simple_t<float, float>(l, a);
    if (!a.u_f32 && window_tiled(a)) return launch_window_prefill_tiled(l, a);
    return a.u_f32 ? simple_t<bf16, float>(l, a) : simple_t<bf16, bf16>(l, a);
}

cudaError_t launch_window_decode(const Launch& l, DenseType type, WindowArgs a, int* launches) {
    if (a.m != 1) return cudaErrorInvalidValue;
    a.u_f32 = 1;
    if (type == kDenseBf16 && !bad_geometry(a) && window_tiled(a)) {
        a.dyn = dev_dyn(l);
        *launches = 1;
        return launch_window_decode_tiled(l, a);
    }
    *launches = 3;
    cudaError_t e = launch_window_append(l, type, a);
    if (e == cudaSuccess) e = launch_window_pool(l, type, a);
    return e == cudaSuccess ? launch_window_attention(l, type, a) : e;
}

}  // namespace smelt
