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
// CTAs and a column over kParts lanes that keep their keys' rows in registers for the whole chunk;
// the chunk's operands pass through shared memory, a stage of positions at a time, two in flight.
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
    pdl_trigger();
    if (state_smem) {  // the last token's state: only this kernel writes it
        for (int i = tid; i < D * D / 4; i += kThreads) cp_async16(ss + 4 * i, state + 4 * i);
        cp_async_commit();
    }
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
    {
        // eight lanes a channel
        const int lane = tid & 7;
        for (int d0 = 0; d0 < D; d0 += kThreads / 8) {
            const int d = d0 + (tid >> 3);
            float acc = 0.f;
            if (d < D) {
                const bf16* w = a.w2 + (size_t)(h * D + d) * a.rank;
                for (int i = lane * 8; i < a.rank; i += 64) {
                    const uint4 v = *reinterpret_cast<const uint4*>(w + i);
                    const uint32_t q[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
                    for (int j = 0; j < 4; ++j) acc = fmaf(__uint_as_float(q[j] & 0xFFFF0000u), st[i + 2 * j + 1], fmaf(__uint_as_float(q[j] << 16), st[i + 2 * j], acc));
                }
            }
            acc += __shfl_xor_sync(0xffffffffu, acc, 4);
            acc += __shfl_xor_sync(0xffffffffu, acc, 2);
            acc += __shfl_xor_sync(0xffffffffu, acc, 1);
            if (d < D && lane == 0) sw[d] = expf(-expf(acc + to_f32(a.w0[h * D + d])));
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
constexpr int kParts = 4;  // lanes a column

// KP: keys of a lane (a multiple of 4, dim <= kParts KP); COLS value columns a CTA.
template <int KP, int COLS>
__global__ void __launch_bounds__(COLS* kParts) wkv_prefill_kernel(const WkvArgs a) {
    constexpr int kStage = KP > 16 ? 8 : 16;  // positions
    constexpr int kPitch = KP + 4;  // parts of a row start in different banks
    constexpr int kRow = kParts * kPitch, kCta = COLS * kParts;
    __shared__ __align__(16) float s_op[2][3][kStage][kRow];  // r, k, w
    __shared__ __align__(16) float s_v[2][kStage][COLS];
    const int D = a.dim, h = blockIdx.y, c0 = blockIdx.x * COLS, tid = threadIdx.x, part = tid % kParts, col = tid / kParts, c = c0 + col;
    const bool live = c < D;
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    for (int i = tid; i < 2 * 3 * kStage * kRow; i += kCta) (&s_op[0][0][0][0])[i] = 0.f;  // keys past dim stay zero
    for (int i = tid; i < 2 * kStage * COLS; i += kCta) (&s_v[0][0][0])[i] = 0.f;
    __syncthreads();

    const int hd = a.heads * D;
    auto issue = [&](int stage) {
        const int t0 = stage * kStage, n = min(kStage, a.m - t0), buf = stage & 1;
        for (int i = tid; i < n * D; i += kCta) {
            const int t = i / D, d = i % D, at = d / KP * kPitch + d % KP;
            const float* u = a.u + (size_t)(t0 + t) * a.ldu + h * D + d;
            cp_async4(&s_op[buf][0][t][at], u);
            cp_async4(&s_op[buf][1][t][at], u + a.group);
            cp_async4(&s_op[buf][2][t][at], a.decay + (size_t)(t0 + t) * hd + h * D + d);
        }
        for (int i = tid; i < n * COLS; i += kCta) {
            const int t = i / COLS, j = i % COLS;
            if (c0 + j < D) cp_async4(&s_v[buf][t][j], a.u + (size_t)(t0 + t) * a.ldu + 2 * a.group + h * D + c0 + j);
        }
        cp_async_commit();
    };
    const int stages = (a.m + kStage - 1) / kStage;
    issue(0);

    float S[KP], ub[KP];
    float* state = a.state + (size_t)h * D * D;
    const bool fresh = dyn_position(a.dyn) == 0u;
#pragma unroll
    for (int j = 0; j < KP; ++j) {
        const int k = part * KP + j;
        ub[j] = k < D ? to_f32(a.bonus[h * D + k]) : 0.f;
        S[j] = live && k < D && !fresh ? state[(size_t)k * D + c] : 0.f;
    }
    float* o = static_cast<float*>(a.out) + h * D + c;
    for (int stage = 0; stage < stages; ++stage) {
        if (stage + 1 < stages) issue(stage + 1);
        else cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const int buf = stage & 1, n = min(kStage, a.m - stage * kStage);
#pragma unroll 2
        for (int t = 0; t < n; ++t) {
            const float4* r4 = reinterpret_cast<const float4*>(&s_op[buf][0][t][part * kPitch]);
            const float4* k4 = reinterpret_cast<const float4*>(&s_op[buf][1][t][part * kPitch]);
            const float4* w4 = reinterpret_cast<const float4*>(&s_op[buf][2][t][part * kPitch]);
            const float v = s_v[buf][t][col];
            float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int q = 0; q < KP / 4; ++q) {
                const float4 r = r4[q], k = k4[q], w = w4[q];
                const float rr[4] = {r.x, r.y, r.z, r.w}, kk[4] = {k.x, k.y, k.z, k.w}, ww[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float kv = kk[j] * v;
                    acc[j] = fmaf(rr[j], fmaf(ub[4 * q + j], kv, S[4 * q + j]), acc[j]);
                    S[4 * q + j] = fmaf(ww[j], S[4 * q + j], kv);
                }
            }
            float sum = (acc[0] + acc[1]) + (acc[2] + acc[3]);
            sum += __shfl_xor_sync(0xffffffffu, sum, 1);
            sum += __shfl_xor_sync(0xffffffffu, sum, 2);
            if (part == 0 && live) o[(size_t)(stage * kStage + t) * hd] = sum;
        }
        __syncthreads();  // the buffer may be refilled
    }
    cp_async_wait<0>();
    if (live)
#pragma unroll
        for (int j = 0; j < KP; ++j)
            if (part * KP + j < D) state[(size_t)(part * KP + j) * D + c] = S[j];
    if (blockIdx.x == 0)
        for (int i = h * kCta + tid; i < a.ld; i += a.heads * kCta) a.before[i] = a.h[(size_t)(a.m - 1) * a.ld + i];
}

// Any dim: one CTA per head, the state read and written in global memory, position after position.
__global__ void __launch_bounds__(kThreads) wkv_prefill_simple_kernel(const WkvArgs a) {
    pdl_trigger();
    pdl_wait();
    if (dyn_skip(a.dyn)) return;
    const int D = a.dim, h = blockIdx.x, hd = a.heads * D;
    const bool fresh = dyn_position(a.dyn) == 0u;
    float* state = a.state + (size_t)h * D * D;
    for (int c = threadIdx.x; c < D; c += kThreads)  // a thread's columns are its own
        for (int t = 0; t < a.m; ++t) {
            const float* u = a.u + (size_t)t * a.ldu + h * D;
            const float v = u[2 * a.group + c];
            float o = 0.f;
            for (int k = 0; k < D; ++k) {
                const float s = fresh && t == 0 ? 0.f : state[(size_t)k * D + c], kv = u[a.group + k] * v;
                o = fmaf(u[k], fmaf(to_f32(a.bonus[h * D + k]), kv, s), o);
                state[(size_t)k * D + c] = fmaf(a.decay[(size_t)t * hd + h * D + k], s, kv);
            }
            static_cast<float*>(a.out)[(size_t)t * hd + h * D + c] = o;
        }
    for (int i = h * kThreads + threadIdx.x; i < a.ld; i += a.heads * kThreads) a.before[i] = a.h[(size_t)(a.m - 1) * a.ld + i];
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

bool bad(const WkvArgs& a) { return a.heads <= 0 || a.dim <= 0 || a.group < a.heads * a.dim || a.m <= 0; }

template <int KP, int COLS>
cudaError_t prefill_t(const Launch& l, const WkvArgs& a) {
    return launch_chained(l, wkv_prefill_kernel<KP, COLS>, dim3((a.dim + COLS - 1) / COLS, a.heads), dim3(COLS * kParts), 0, a);
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
    if (a.dim <= 16) return prefill_t<4, 16>(l, a);
    if (a.dim <= 32) return prefill_t<8, 16>(l, a);
    if (a.dim <= 64) return prefill_t<16, 16>(l, a);
    if (a.dim <= 128) return prefill_t<32, 16>(l, a);
    return launch_chained(l, wkv_prefill_simple_kernel, dim3(a.heads), dim3(kThreads), 0, a);
}

cudaError_t launch_wkv_gate_rows(const Launch& l, DenseType type, WkvArgs a) {
    if (bad(a) || a.ldz < a.heads * a.dim) return cudaErrorInvalidValue;
    a.dyn = dev_dyn(l);
    const dim3 grid(a.m, (a.heads + kWarps - 1) / kWarps), block(kThreads);
    return type == kDenseF32 ? launch_chained(l, wkv_gate_rows_kernel<float>, grid, block, 0, a) : launch_chained(l, wkv_gate_rows_kernel<bf16>, grid, block, 0, a);
}

}  // namespace smelt
