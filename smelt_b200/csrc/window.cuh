// What the window + pooled-block attention kernels share: which keys a position sees, the block
// mean, and the softmax weight of a softcapped score.
#pragma once
#include <cmath>

#include "dense.h"

namespace smelt {

// The blocks a query at position i sees: [0, n).
__device__ __forceinline__ uint32_t visible_blocks(uint32_t i, uint32_t window, uint32_t pool) { return i + 1u >= window ? (i + 1u - window) / pool : 0u; }
__device__ __forceinline__ uint32_t window_start(uint32_t i, uint32_t window) { return i + 1u > window ? i + 1u - window : 0u; }


// Mean of a block's rows as the cache holds them, in position order.
template <class TC>
__device__ __forceinline__ float block_mean(const TC* head, uint32_t first, uint32_t pool, uint32_t ring, int pitch, int d) {
    float sum = 0.f;
    uint32_t slot = first % ring;
    for (uint32_t j = 0; j < pool; ++j) {
        sum += to_f32(head[(size_t)slot * pitch + d]);
        slot = slot + 1u == ring ? 0u : slot + 1u;
    }
    return sum / (float)pool;
}

// A softcapped score is bounded, so its exponential needs no running maximum: every weight is
// taken relative to one reference (0, or softcap - 64 where exp(softcap) could overflow a sum),
// and partial sums of different keys simply add.  With y = exp(2 s / softcap),
// softcap tanh(s / softcap) = softcap - 2 softcap / (y + 1); the weight is 2 to the power of that
// in units of log2(e).  The sink's weight is exp(-reference).
struct CapWeight {
    float rate;   // y = 2^(dot * rate)
    float top, span;  // weight = 2^(top - span / (y + 1))
    float sink;
};
constexpr float kMaxTiledCap = 128.f;  // beyond it the sink's weight would underflow
inline CapWeight cap_weight(float scale, float softcap) {
    const double log2e = 1.4426950408889634, ref = softcap > 64.f ? softcap - 64.0 : 0.0;
    return CapWeight{(float)(2.0 * scale / softcap * log2e), (float)((softcap - ref) * log2e), (float)(2.0 * softcap * log2e), (float)exp(-ref)};
}
__device__ __forceinline__ float rcp_approx(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float cap_weight_of(const CapWeight& w, float dot) { return exp2_approx(fmaf(-w.span, rcp_approx(exp2_approx(dot * w.rate) + 1.f), w.top)); }

// Shapes and softcaps the tensor-core kernels take.
inline bool window_tiled(const WindowArgs& a) { return a.kp <= 256 && a.vp <= 256 && a.softcap > 0.f && a.softcap <= kMaxTiledCap; }
cudaError_t launch_window_prefill_tiled(const Launch& l, const WindowArgs& a);
cudaError_t launch_window_decode_tiled(const Launch& l, const WindowArgs& a);

}  // namespace smelt
