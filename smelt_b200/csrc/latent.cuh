// What the latent attention kernels share: rotation of adjacent pairs by exact angles.
#pragma once
#include "stack.h"

namespace smelt {

// cos and sin of position * freq: product and reduction to one turn in fp64, then fp32.
__device__ __forceinline__ float2 rotary_cos_sin(uint32_t position, double freq) {
    const double a = (double)position * freq, turns = rint(a * 0.15915494309189535);
    float s, c;
    sincosf((float)fma(-turns, 6.283185307179586, a), &s, &c);
    return make_float2(c, s);
}

// Element i of the vector v with its first `dims` elements rotated in pairs (2j, 2j + 1).
template <class T>
__device__ __forceinline__ float rotated(const T* v, int i, int dims, const double* freq, uint32_t position) {
    const float x = to_f32(v[i]);
    if (i >= dims) return x;
    const float2 cs = rotary_cos_sin(position, freq[i >> 1]);
    const float other = to_f32(v[i ^ 1]);
    return i & 1 ? fmaf(x, cs.x, other * cs.y) : fmaf(x, cs.x, -other * cs.y);
}

}  // namespace smelt
