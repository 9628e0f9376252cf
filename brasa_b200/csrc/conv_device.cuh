// What the recurrent mixers share: the short causal convolution over time with its silu, gates, and asynchronous copies.
//
// The inputs of a convolution of `taps` taps that lie before a run are kept in a ring of `taps` rows, position p in row p % taps
// (one more row than needed, so that a step can store its own row while others still read the older ones).
#pragma once
#include "tc_device.cuh"

namespace brasa_dev {

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
// for results that are rounded to bf16
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// The convolution of one channel at token t: x f32 [tokens][ldx] holds this run's inputs, the ring the ones before it.
// ch: the channel in the ring (q channels, then k's, then v's).
struct ConvView {
    const float *ring;
    uint32_t channels, taps, pos0;
};
__device__ __forceinline__ float conv_at(const float *x, uint32_t ldx, uint32_t c, const float *w, uint32_t t, const ConvView &cv, uint32_t ch) {
    float s = 0.0f;
    for (uint32_t i = 0; i < cv.taps; ++i) {
        const uint32_t back = cv.taps - 1 - i;  // tokens before this one
        float v;
        if (back <= t) v = x[(size_t)(t - back) * ldx + c];
        else if (back <= cv.pos0 + t) v = cv.ring[(size_t)((cv.pos0 + t - back) % cv.taps) * cv.channels + ch];
        else v = 0.0f;
        s = fmaf(v, w[(size_t)c * cv.taps + i], s);
    }
    return s;
}

// The same for one token (x its inputs, slot = pos0 % taps); up to four taps with every load on its way at once.
__device__ __forceinline__ float conv_step(const float *x, uint32_t c, const float *w, const ConvView &cv, uint32_t slot, uint32_t ch) {
    if (cv.taps > 4) return conv_at(x, 0, c, w, 0, cv, ch);
    float v[4], k[4];
#pragma unroll
    for (uint32_t b = 0; b < 4; ++b) {  // b tokens before this one
        const bool live = b < cv.taps && b <= cv.pos0;
        v[b] = !live ? 0.0f : (b == 0 ? x[c] : cv.ring[(size_t)(slot >= b ? slot - b : slot + cv.taps - b) * cv.channels + ch]);
        k[b] = b < cv.taps ? w[(size_t)c * cv.taps + cv.taps - 1 - b] : 0.0f;
    }
    return fmaf(v[0], k[0], fmaf(v[1], k[1], fmaf(v[2], k[2], v[3] * k[3])));
}

// convolution, bias and silu of one channel for tokens t0 .. t0 + n - 1 (n up to CONV_RUN), handed to put(t, value)
constexpr uint32_t CONV_RUN = 16;
template <bool FAST = false, typename Put>
__device__ __forceinline__ void conv_chunk(const float *x, uint32_t ldx, uint32_t c, const float *w, float bias, uint32_t t0, uint32_t n, const ConvView &cv, uint32_t ch, Put put) {
    if (cv.taps <= 4) {  // the window in registers
        float wr[4], xr[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int tap = (int)cv.taps - 4 + i, back = 4 - i;  // xr[i]: `back` tokens before t0
            wr[i] = tap >= 0 ? w[(size_t)c * cv.taps + tap] : 0.0f;
            xr[i] = 0.0f;
            if (i > 0 && tap > 0) {  // xr[1 .. 3] hold the three tokens ahead of the first one, where the window reaches them
                const uint32_t bk = back;
                if (bk <= t0) xr[i] = x[(size_t)(t0 - bk) * ldx + c];
                else if (bk <= cv.pos0 + t0) xr[i] = cv.ring[(size_t)((cv.pos0 + t0 - bk) % cv.taps) * cv.channels + ch];
            }
        }
        float in[CONV_RUN];
#pragma unroll
        for (uint32_t t = 0; t < CONV_RUN; ++t) in[t] = t < n ? x[(size_t)(t0 + t) * ldx + c] : 0.0f;
#pragma unroll
        for (uint32_t t = 0; t < CONV_RUN; ++t) {
            xr[0] = xr[1];
            xr[1] = xr[2];
            xr[2] = xr[3];
            xr[3] = in[t];
            const float z = fmaf(xr[3], wr[3], fmaf(xr[2], wr[2], fmaf(xr[1], wr[1], fmaf(xr[0], wr[0], bias))));
            if (t < n) put(t, FAST ? silu_fast(z) : silu_f(z));
        }
    } else {
        for (uint32_t t = 0; t < n; ++t) put(t, silu_f(conv_at(x, ldx, c, w, t0 + t, cv, ch) + bias));
    }
}

__device__ __forceinline__ void cp4(float *dst, const float *src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp16(void *dst, const void *src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

}  // namespace brasa_dev
