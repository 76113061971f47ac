// RWKV-style time mixing: token shift, decay, the matrix-valued recurrence, gate.
//
// Per head, with S[key][value]:  o = (S + diag(u) k v^T)^T r;  S <- diag(w) S + k v^T;
// w = exp(-exp(W2 tanh(inner) + w0)); z = o / rms(o) * norm * silu(g).  All in fp32; the state stays
// in fp32 from token to token, and counts as zero at position 0, so nothing is cleared between
// sequences.
//
// wkv_decode_kernel: one CTA per head, the whole step behind the projections.  The state and the
// head's rows of W2, which do not depend on the launch in front, are requested before the wait for
// it.  wkv_prefill_kernel: value columns are independent, so the columns of a head are cut over
// CTAs, and the keys over sixteen lanes that keep their part of four columns in registers for the
// whole chunk (packed fp32 pairs); the chunk's operands pass through shared memory, a stage of
// positions at a time, two in flight.
#include <algorithm>

#include "stack.h"

namespace smelt {

namespace {

constexpr int kThreads = 256, kWarps = kThreads / 32;

__device__ __forceinline__ float cta_sum(float v, float* scratch) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) tot += scratch[w];
    return tot;
}

// VEC: value columns a thread takes (4 where dim is a multiple of 4, else 1); the state's rows are cut over the thread groups.
template <int VEC>
__global__ void __launch_bounds__(kThreads) wkv_decode_kernel(const WkvArgs a, int state_smem) {
    extern __shared__ __align__(16) float smem[];
    __shared__ float s_sum[2][kWarps];
    const int D = a.dim, h = blockIdx.x, tid = threadIdx.x, cols = D / VEC, groups = min(kThreads / cols, D);
    float *sr = smem, *sk = sr + D, *sv = sk + D, *sw = sv + D, *st = sw + D;  // st: tanh of the decay's inner values [rank]
    float* so = st + a.rank;                                                  // [groups][D]
    float* ss = smem + ((4 * D + a.rank + groups * D + 3) & ~3);              // [D][D] where it fits
    float* state = a.state + (size_t)h * D * D;
    if (state_smem) {  // the last token's state: only this kernel writes it
        for (int i = tid; i < D * D / 4; i += kThreads) cp_async16(ss + 4 * i, state + 4 * i);
        cp_async_commit();
    }
    // W2: eight lanes a channel, 64 inner values a piece; the first pieces are held in registers
    constexpr int kHeld = 4;
    const int pieces = a.rank / 64, passes = (D + kThreads / 8 - 1) / (kThreads / 8), lane8 = tid & 7;
    auto w2_piece = [&](int n) {
        const int d = n / pieces * (kThreads / 8) + (tid >> 3);
        return d < D ? *reinterpret_cast<const uint4*>(a.w2 + (size_t)(h * D + d) * a.rank + n % pieces * 64 + lane8 * 8) : make_uint4(0, 0, 0, 0);
    };
    uint4 held[kHeld];
#pragma unroll
    for (int n = 0; n < kHeld; ++n) held[n] = n < passes * pieces ? w2_piece(n) : make_uint4(0, 0, 0, 0);
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) {
        cp_async_wait<0>();
        return;
    }
    const bool fresh = dyn_position(a.dyn) == 0u;
    const float* u = a.u;
    float ruk = 0.f;
    for (int d = tid; d < D; d += kThreads) {
        const int c = h * D + d;
        const float r = u[c], k = u[a.group + c];
        sr[d] = r; sk[d] = k; sv[d] = u[2 * a.group + c];
        ruk = fmaf(r * to_f32(a.bonus[c]), k, ruk);
    }
    for (int i = tid; i < a.rank; i += kThreads) st[i] = tanhf(u[4 * a.group + i]);
    ruk = cta_sum(ruk, s_sum[0]);  // with a barrier: st is ready
    float inner = 0.f;
    for (int n0 = 0; n0 < passes * pieces; n0 += kHeld) {
#pragma unroll
        for (int j = 0; j < kHeld; ++j) {
            const int n = n0 + j;
            if (n >= passes * pieces) break;
            const uint4 v = n0 == 0 ? held[j] : w2_piece(n);
            const float* t = st + n % pieces * 64 + lane8 * 8;
            const uint32_t q[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
            for (int i = 0; i < 4; ++i) inner = fmaf(__uint_as_float(q[i] & 0xFFFF0000u), t[2 * i + 1], fmaf(__uint_as_float(q[i] << 16), t[2 * i], inner));
            if (n % pieces != pieces - 1) continue;
            inner += __shfl_xor_sync(0xffffffffu, inner, 4);
            inner += __shfl_xor_sync(0xffffffffu, inner, 2);
            inner += __shfl_xor_sync(0xffffffffu, inner, 1);
            const int d = n / pieces * (kThreads / 8) + (tid >> 3);
            if (d < D && lane8 == 0) sw[d] = expf(-expf(inner + to_f32(a.w0[h * D + d])));
            inner = 0.f;
        }
    }
    cp_async_wait<0>();
    __syncthreads();
    const int col = tid % cols * VEC, grp = tid / cols;
    if (grp < groups) {
        float o[VEC], v[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) { o[j] = 0.f; v[j] = sv[col + j]; }
        const float* from = state_smem ? ss : state;
#pragma unroll 4
        for (int k = grp; k < D; k += groups) {
            float s[VEC];
            if constexpr (VEC == 4) {
                const float4 t = *reinterpret_cast<const float4*>(from + (size_t)k * D + col);
                s[0] = t.x; s[1] = t.y; s[2] = t.z; s[3] = t.w;
            } else {
                s[0] = from[(size_t)k * D + col];
            }
            const float r = sr[k], kk = sk[k], w = sw[k];
#pragma unroll
            for (int j = 0; j < VEC; ++j) {
                if (fresh) s[j] = 0.f;
                o[j] = fmaf(r, s[j], o[j]);
                s[j] = fmaf(w, s[j], kk * v[j]);
            }
            if constexpr (VEC == 4) *reinterpret_cast<float4*>(state + (size_t)k * D + col) = make_float4(s[0], s[1], s[2], s[3]);
            else state[(size_t)k * D + col] = s[0];
        }
#pragma unroll
        for (int j = 0; j < VEC; ++j) so[grp * D + col + j] = o[j];
    }
    __syncthreads();
    float sq = 0.f;
    for (int d = tid; d < D; d += kThreads) {
        float o = ruk * sv[d];
        for (int g = 0; g < groups; ++g) o += so[g * D + d];
        so[d] = o;  // this thread alone reads the column
        sq = fmaf(o, o, sq);
    }
    const float f = rsqrtf(cta_sum(sq, s_sum[1]) / (float)D + a.eps);
    float* z = static_cast<float*>(a.out);
    for (int d = tid; d < D; d += kThreads) {
        const int c = h * D + d;
        z[c] = so[d] * f * to_f32(a.norm[c]) * silu(u[3 * a.group + c]);
    }
    for (int i = h * kThreads + tid; i < a.ld; i += a.heads * kThreads) a.before[i] = a.h[i];
}

// out[s][r] = h + (h of the row before - h) mu[s]
template <class T>
__global__ void __launch_bounds__(kThreads) shift_mix_rows_kernel(const WkvArgs a) {
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    const int r = blockIdx.x;
    const bool zero = r == 0 && dyn_position(a.dyn) == 0u;
    const float* h = a.h + (size_t)r * a.ld;
    const float* b = r > 0 ? h - a.ld : a.before;
    T* out = static_cast<T*>(a.out);
    for (int i = threadIdx.x * 4; i < a.ld; i += kThreads * 4) {
        const float4 v = *reinterpret_cast<const float4*>(h + i), p = zero ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(b + i);
#pragma unroll
        for (int s = 0; s < 5; ++s) {
            const uint2 m = *reinterpret_cast<const uint2*>(a.mu + (size_t)s * a.ld + i);
            const float4 x = make_float4(fmaf(p.x - v.x, __uint_as_float(m.x << 16), v.x), fmaf(p.y - v.y, __uint_as_float(m.x & 0xFFFF0000u), v.y),
                                         fmaf(p.z - v.z, __uint_as_float(m.y << 16), v.z), fmaf(p.w - v.w, __uint_as_float(m.y & 0xFFFF0000u), v.w));
            T* dst = out + ((size_t)s * a.m + r) * a.ld + i;
            if constexpr (sizeof(T) == 4) {
                *reinterpret_cast<float4*>(dst) = x;
            } else {
                const __nv_bfloat162 lo = __floats2bfloat162_rn(x.x, x.y), hi = __floats2bfloat162_rn(x.z, x.w);
                *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
            }
        }
    }
}

// ── prompt chunk ────────────────────────────────────────────────────────────
// Two fp32 values in one register pair.
__device__ __forceinline__ uint64_t pair2(float x, float y) {
    uint64_t v;
    asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(x), "f"(y));
    return v;
}
__device__ __forceinline__ float2 halves(uint64_t v) {
    float2 f;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
    return f;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}

constexpr int kParts = 16, kLaneCols = 4, kPrefillThreads = 64, kPrefillCols = kPrefillThreads / kParts * kLaneCols, kTogether = 4;

// KP keys (a multiple of 4, dim <= kParts KP) and kLaneCols value columns a lane; lane p of sixteen has the keys 64 q + 4 p + 0..3.
// The bonus adds sum(r u k) v, its sum taken along with the others.  Four positions' sums over the
// sixteen lanes are reduced together: sixteen values, halved with every exchange.
template <int KP>
__global__ void __launch_bounds__(kPrefillThreads) wkv_prefill_kernel(const WkvArgs a) {
    constexpr int kStage = 64 / KP, kRow = kParts * KP, kQ = KP / 4;
    __shared__ __align__(16) float s_op[2][3][kStage][kRow];  // r, k, w
    __shared__ __align__(16) float s_v[2][kStage][kPrefillCols];
    const int D = a.dim, h = blockIdx.y, c0 = blockIdx.x * kPrefillCols, tid = threadIdx.x, part = tid % kParts, group = tid / kParts, col = c0 + group * kLaneCols;
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    for (int i = tid; i < 2 * 3 * kStage * kRow; i += kPrefillThreads) (&s_op[0][0][0][0])[i] = 0.f;  // keys past dim stay zero
    for (int i = tid; i < 2 * kStage * kPrefillCols; i += kPrefillThreads) (&s_v[0][0][0])[i] = 0.f;
    __syncthreads();

    const int hd = a.heads * D;
    const bool wide = D % 4 == 0 && a.ldu % 4 == 0 && a.group % 4 == 0;  // rows of whole 16-byte pieces
    auto issue = [&](int stage) {
        const int t0 = stage * kStage, n = min(kStage, a.m - t0), buf = stage & 1;
        const float* u0 = a.u + (size_t)t0 * a.ldu + h * D;
        const float* w0 = a.decay + (size_t)t0 * hd + h * D;
        if (wide) {
            const int pieces = D / 4;
            for (int i = tid; i < n * pieces; i += kPrefillThreads) {
                const int t = i / pieces, d = 4 * (i - t * pieces);
                const float* u = u0 + (size_t)t * a.ldu + d;
                cp_async16(&s_op[buf][0][t][d], u);
                cp_async16(&s_op[buf][1][t][d], u + a.group);
                cp_async16(&s_op[buf][2][t][d], w0 + (size_t)t * hd + d);
            }
            for (int i = tid; i < n * (kPrefillCols / 4); i += kPrefillThreads) {
                const int t = i / (kPrefillCols / 4), j = i % (kPrefillCols / 4) * 4;
                if (c0 + j < D) cp_async16(&s_v[buf][t][j], u0 + (size_t)t * a.ldu + 2 * a.group + c0 + j);
            }
        } else {
            for (int i = tid; i < n * D; i += kPrefillThreads) {
                const int t = i / D, d = i - t * D;
                const float* u = u0 + (size_t)t * a.ldu + d;
                cp_async4(&s_op[buf][0][t][d], u);
                cp_async4(&s_op[buf][1][t][d], u + a.group);
                cp_async4(&s_op[buf][2][t][d], w0 + (size_t)t * hd + d);
            }
            for (int i = tid; i < n * kPrefillCols; i += kPrefillThreads) {
                const int t = i / kPrefillCols, j = i % kPrefillCols;
                if (c0 + j < D) cp_async4(&s_v[buf][t][j], u0 + (size_t)t * a.ldu + 2 * a.group + c0 + j);
            }
        }
        cp_async_commit();
    };
    const int stages = (a.m + kStage - 1) / kStage;
    issue(0);

    uint64_t S[kLaneCols][KP / 2], ub[KP / 2];
    float* state = a.state + (size_t)h * D * D;
    const bool fresh = dyn_position(a.dyn) == 0u;
#pragma unroll
    for (int i = 0; i < KP / 2; ++i) {
        const int k = i / 2 * 64 + part * 4 + i % 2 * 2;
        auto bonus = [&](int j) { return j < D ? to_f32(a.bonus[h * D + j]) : 0.f; };
        ub[i] = pair2(bonus(k), bonus(k + 1));
#pragma unroll
        for (int c = 0; c < kLaneCols; ++c) {
            auto at = [&](int j) { return j < D && col + c < D && !fresh ? state[(size_t)j * D + col + c] : 0.f; };
            S[c][i] = pair2(at(k), at(k + 1));
        }
    }
    float* o = static_cast<float*>(a.out) + h * D;
    for (int stage = 0; stage < stages; ++stage) {
        if (stage + 1 < stages) issue(stage + 1);
        else cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const int buf = stage & 1, n = min(kStage, a.m - stage * kStage);
        for (int t = 0; t < n; t += kTogether) {
            float sum[kTogether * kLaneCols];
            auto position = [&](int x) {
                const ulonglong2* r2 = reinterpret_cast<const ulonglong2*>(&s_op[buf][0][t + x][part * 4]);
                const ulonglong2* k2 = reinterpret_cast<const ulonglong2*>(&s_op[buf][1][t + x][part * 4]);
                const ulonglong2* w2 = reinterpret_cast<const ulonglong2*>(&s_op[buf][2][t + x][part * 4]);
                const float4 v4 = *reinterpret_cast<const float4*>(&s_v[buf][t + x][group * kLaneCols]);
                const float v[kLaneCols] = {v4.x, v4.y, v4.z, v4.w};
                uint64_t acc[kLaneCols], b = 0;
#pragma unroll
                for (int q = 0; q < kQ; ++q) {
                    const ulonglong2 r = r2[q * 16], k = k2[q * 16], w = w2[q * 16];
                    const uint64_t rr[2] = {r.x, r.y}, kk[2] = {k.x, k.y}, ww[2] = {w.x, w.y};
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        const int i = 2 * q + j;
                        const uint64_t ru = mul2(rr[j], ub[i]);
                        b = i == 0 ? mul2(ru, kk[j]) : fma2(ru, kk[j], b);
#pragma unroll
                        for (int c = 0; c < kLaneCols; ++c) {
                            acc[c] = i == 0 ? mul2(rr[j], S[c][i]) : fma2(rr[j], S[c][i], acc[c]);
                            S[c][i] = fma2(ww[j], S[c][i], mul2(kk[j], pair2(v[c], v[c])));
                        }
                    }
                }
                const float2 bs = halves(b);
#pragma unroll
                for (int c = 0; c < kLaneCols; ++c) {
                    const float2 f = halves(acc[c]);
                    sum[x * kLaneCols + c] = fmaf(bs.x + bs.y, v[c], f.x + f.y);
                }
            };
            if (t + kTogether <= n) {
#pragma unroll
                for (int x = 0; x < kTogether; ++x) position(x);
            } else {
#pragma unroll
                for (int x = 0; x < kTogether; ++x) {
                    if (t + x < n) position(x);
                    else
#pragma unroll
                        for (int c = 0; c < kLaneCols; ++c) sum[x * kLaneCols + c] = 0.f;
                }
            }
#pragma unroll
            for (int off = kParts / 2; off > 0; off >>= 1) {
                const bool up = part & off;
#pragma unroll
                for (int i = 0; i < off; ++i) {
                    const float keep = up ? sum[i + off] : sum[i], send = up ? sum[i] : sum[i + off];
                    sum[i] = keep + __shfl_xor_sync(0xffffffffu, send, off);
                }
            }
            const int x = part / kLaneCols, c = col + part % kLaneCols;  // the lane's own sum
            if (t + x < n && c < D) o[(size_t)(stage * kStage + t + x) * hd + c] = sum[0];
        }
        __syncthreads();  // the buffer may be refilled
    }
    cp_async_wait<0>();
#pragma unroll
    for (int i = 0; i < KP / 2; ++i) {
        const int k = i / 2 * 64 + part * 4 + i % 2 * 2;
#pragma unroll
        for (int c = 0; c < kLaneCols; ++c) {
            const float2 f = halves(S[c][i]);
            if (col + c < D) {
                if (k < D) state[(size_t)k * D + col + c] = f.x;
                if (k + 1 < D) state[(size_t)(k + 1) * D + col + c] = f.y;
            }
        }
    }
    if (blockIdx.x == 0)
        for (int i = h * kPrefillThreads + tid; i < a.ld; i += a.heads * kPrefillThreads) a.before[i] = a.h[(size_t)(a.m - 1) * a.ld + i];
}

// One warp per (row, head).
template <class T>
__global__ void __launch_bounds__(kThreads) wkv_gate_rows_kernel(const WkvArgs a) {
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    const int r = blockIdx.x, h = blockIdx.y * kWarps + (threadIdx.x >> 5), lane = threadIdx.x & 31, D = a.dim;
    if (h >= a.heads) return;
    const float* o = a.o + ((size_t)r * a.heads + h) * D;
    const float* g = a.u + (size_t)r * a.ldu + 3 * a.group + h * D;
    T* z = static_cast<T*>(a.out) + (size_t)r * a.ldz + h * D;
    float ss = 0.f;
    for (int d = lane; d < D; d += 32) ss = fmaf(o[d], o[d], ss);
    const float f = rsqrtf(warp_sum(ss) / (float)D + a.eps);
    for (int d = lane; d < D; d += 32) z[d] = from_f32<T>(o[d] * f * to_f32(a.norm[h * D + d]) * silu(g[d]));
}

// The same for a dim of 4 LANES: LANES lanes a head, four elements a lane, one CTA per row.
template <class T, int LANES>
__global__ void __launch_bounds__(kThreads) wkv_gate_vector_kernel(const WkvArgs a) {
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    const int r = blockIdx.x, hd = a.heads * 4 * LANES;
    const float* o = a.o + (size_t)r * hd;
    const float* g = a.u + (size_t)r * a.ldu + 3 * a.group;
    T* z = static_cast<T*>(a.out) + (size_t)r * a.ldz;
    for (int base = 0; base < hd; base += 4 * kThreads) {  // whole warps take part in the sums
        const int i = base + 4 * threadIdx.x;
        const bool in = i < hd;
        const float4 v = in ? *reinterpret_cast<const float4*>(o + i) : make_float4(0.f, 0.f, 0.f, 0.f), y = in ? *reinterpret_cast<const float4*>(g + i) : v;
        const uint2 n = in ? *reinterpret_cast<const uint2*>(a.norm + i) : make_uint2(0, 0);
        float ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)));
#pragma unroll
        for (int off = LANES / 2; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
        if (!in) continue;
        const float f = rsqrtf(ss / (float)(4 * LANES) + a.eps);
        const float4 w = make_float4(v.x * f * __uint_as_float(n.x << 16) * silu(y.x), v.y * f * __uint_as_float(n.x & 0xFFFF0000u) * silu(y.y),
                                     v.z * f * __uint_as_float(n.y << 16) * silu(y.z), v.w * f * __uint_as_float(n.y & 0xFFFF0000u) * silu(y.w));
        if constexpr (sizeof(T) == 4) {
            *reinterpret_cast<float4*>(z + i) = w;
        } else {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(w.x, w.y), hi = __floats2bfloat162_rn(w.z, w.w);
            *reinterpret_cast<uint2*>(z + i) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
        }
    }
}

template <class T>
cudaError_t gate_t(const Launch& l, const WkvArgs& a) {
    if (a.ldz % 4 == 0 && a.ldu % 4 == 0) {
        if (a.dim == 32) return launch_chained(l, wkv_gate_vector_kernel<T, 8>, dim3(a.m), dim3(kThreads), 0, a);
        if (a.dim == 64) return launch_chained(l, wkv_gate_vector_kernel<T, 16>, dim3(a.m), dim3(kThreads), 0, a);
        if (a.dim == 128) return launch_chained(l, wkv_gate_vector_kernel<T, 32>, dim3(a.m), dim3(kThreads), 0, a);
    }
    return launch_chained(l, wkv_gate_rows_kernel<T>, dim3(a.m, (a.heads + kWarps - 1) / kWarps), dim3(kThreads), 0, a);
}

bool bad(const WkvArgs& a) { return a.heads <= 0 || a.dim <= 0 || a.group < a.heads * a.dim || a.m <= 0; }

template <int KP>
cudaError_t prefill_t(const Launch& l, const WkvArgs& a) {
    return launch_chained(l, wkv_prefill_kernel<KP>, dim3((a.dim + kPrefillCols - 1) / kPrefillCols, a.heads), dim3(kPrefillThreads), 0, a);
}

}  // namespace

cudaError_t launch_wkv_decode(const Launch& l, WkvArgs a) {
    if (bad(a) || a.rank <= 0 || a.rank % 64 || a.dim > 1024) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    const int vec = a.dim % 4 == 0 ? 4 : 1, cols = a.dim / vec;
    if (cols > kThreads) return cudaErrorInvalidValue;
    const int groups = std::min(kThreads / cols, a.dim);
    size_t smem = (size_t)((4 * a.dim + a.rank + groups * a.dim + 3) & ~3) * sizeof(float);
    const size_t with_state = smem + (size_t)a.dim * a.dim * sizeof(float);
    const int staged = vec == 4 && with_state <= 200 * 1024 ? 1 : 0;
    if (staged) smem = with_state;
    return vec == 4 ? launch_chained(l, wkv_decode_kernel<4>, dim3(a.heads), dim3(kThreads), smem, a, staged) : launch_chained(l, wkv_decode_kernel<1>, dim3(a.heads), dim3(kThreads), smem, a, 0);
}

cudaError_t launch_shift_mix_rows(const Launch& l, DenseType type, WkvArgs a) {
    if (a.ld <= 0 || a.ld % 4 || a.m <= 0) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    return type == kDenseF32 ? launch_chained(l, shift_mix_rows_kernel<float>, dim3(a.m), dim3(kThreads), 0, a) : launch_chained(l, shift_mix_rows_kernel<bf16>, dim3(a.m), dim3(kThreads), 0, a);
}

cudaError_t launch_wkv_prefill(const Launch& l, WkvArgs a) {
    if (bad(a)) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    if (a.dim <= 64) return prefill_t<4>(l, a);
    if (a.dim <= 128) return prefill_t<8>(l, a);
    return a.dim <= 256 ? prefill_t<16>(l, a) : cudaErrorInvalidValue;
}

cudaError_t launch_wkv_gate_rows(const Launch& l, DenseType type, WkvArgs a) {
    if (bad(a) || a.ldz < a.heads * a.dim) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    return type == kDenseF32 ? gate_t<float>(l, a) : gate_t<bf16>(l, a);
}

}  // namespace smelt
