// Prefill attention inside a sliding window (window_attn.h): score = (q_own . k_head + q_shared . k_shared) * scale, optionally
// softcapped, softmax over the visible keys, output times sigmoid(gate of the head).
//
// window_tc_kernel (bf16, tcgen05): one CTA = 128 queries of one head, 128-key tiles from the first tile its window touches.
// Warp 8 (one lane) fetches K, shared-K and V tiles by TMA and issues every product; warps 0-7 are the softmax, two threads
// per query row. S of tile j + 1 is computed while the probabilities of tile j are formed. The probabilities enter P V out
// of tensor memory as two bf16 terms (hi + lo), so the weights keep 16 significant bits and more. One sweep over the keys: a row's
// reference value moves only when a tile exceeds it by more than 8 ln 2, as in the causal kernel of flash_tc.cu. Softcapped
// scores are bounded, so their reference value is 0 throughout: one look at the scores, no maxima, nothing is ever rescaled.
// window_simt_kernel<T>: the same in f32 FMA, for the 32-bit mode and for sizes TMA cannot address.
#include "tc_device.cuh"
#include "window_attn.h"

using namespace brasa_dev;

namespace {

constexpr float LOG2E = 1.4426950408889634f;

// element e of a head's rotated query part, rotated
__device__ __forceinline__ float rotated(const float *q, uint32_t e, uint32_t dims, const float *c, const float *s) {
    const uint32_t half = dims / 2;
    if (e < half) return q[e] * c[e] - q[e + half] * s[e];
    if (e < dims) return q[e] * c[e - half] + q[e - half] * s[e - half];
    return q[e];
}

// ---- f32 FMA: block = 16 queries of one head, tiles of 32 keys ---------------------------------------------------------
constexpr int SQ = 16, SKT = 32, SIMT_VMAX = 16;  // value dims per thread: vdim up to 256

template <typename T>
__global__ void __launch_bounds__(256) window_simt_kernel(WindowAttn a) {
    extern __shared__ __align__(16) float sm[];
    const uint32_t dq = a.dim + a.rot, ldk = dq + 1;
    float *qs = sm, *ks = qs + SQ * dq, *vs = ks + SKT * ldk, *ps = vs + SKT * a.vdim;
    const uint32_t h = blockIdx.y, t0 = blockIdx.x * SQ, tid = threadIdx.x, qi = tid >> 4, l = tid & 15;
    const uint32_t half = a.rot_dims / 2;
    pdl_wait();
    pdl_launch();
    for (uint32_t i = tid; i < SQ * dq; i += 256) {
        const uint32_t t = i / dq, e = i - t * dq;
        float v = 0.0f;
        if (t0 + t < a.tokens) {
            const float *q = a.q + (size_t)(t0 + t) * a.ldq + h * dq;
            const uint32_t p = a.pos0 + t0 + t;
            const float *ct = a.cos_t + (size_t)p * half, *st = a.sin_t + (size_t)p * half;
            if (a.rot == 0) v = rotated(q, e, a.rot_dims, ct, st);
            else v = e < a.dim ? q[e] : rotated(q + a.dim, e - a.dim, a.rot_dims, ct, st);
        }
        qs[i] = v;
    }
    float acc[SIMT_VMAX] = {}, m = -INFINITY, lsum = 0.0f;
    const uint32_t first = a.pos0 + t0, last = a.pos0 + min(t0 + SQ, a.tokens) - 1, lo = max(a.key0, first + 1 > a.window ? first + 1 - a.window : 0u);
    const uint32_t pos = a.pos0 + t0 + qi, kvh = h / (a.heads / a.kv_heads);
    auto row_of = [&](uint32_t p) { return (size_t)(a.ring ? p % a.ring : p - a.key0); };
    for (uint32_t j0 = lo; j0 <= last; j0 += SKT) {
        __syncthreads();
        for (uint32_t i = tid; i < SKT * dq; i += 256) {
            const uint32_t j = i / dq, e = i - j * dq;
            float v = 0.0f;
            if (j0 + j <= last)
                v = e < a.dim ? elem_load((const T *)a.k + row_of(j0 + j) * a.ldk + kvh * a.kstep + e) : elem_load((const T *)a.kr + row_of(j0 + j) * a.ldr + e - a.dim);
            ks[j * ldk + e] = v;
        }
        for (uint32_t i = tid; i < SKT * a.vdim; i += 256) {
            const uint32_t j = i / a.vdim, e = i - j * a.vdim;
            vs[i] = j0 + j <= last ? elem_load((const T *)a.v + row_of(j0 + j) * a.ldv + kvh * a.vstep + e) : 0.0f;
        }
        __syncthreads();
        float s[2] = {0.0f, 0.0f};
        for (uint32_t e = 0; e < dq; ++e) {
            const float q = qs[qi * dq + e];
            s[0] = fmaf(q, ks[l * ldk + e], s[0]);
            s[1] = fmaf(q, ks[(l + 16) * ldk + e], s[1]);
        }
        float mx = -INFINITY;
        for (int u = 0; u < 2; ++u) {
            const uint32_t j = j0 + l + 16 * u;
            s[u] *= a.scale;
            if (a.softcap > 0.0f) s[u] = a.softcap * tanhf(s[u] / a.softcap);
            if (j > pos || pos - j >= a.window) s[u] = -INFINITY;
            mx = fmaxf(mx, s[u]);
        }
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        const float mn = fmaxf(m, mx), r = m == -INFINITY ? 0.0f : expf(m - mn);
        float sum = 0.0f;
        for (int u = 0; u < 2; ++u) {
            const float p = s[u] == -INFINITY ? 0.0f : expf(s[u] - mn);
            ps[qi * SKT + l + 16 * u] = p;
            sum += p;
        }
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        lsum = lsum * r + sum;
        m = mn;
        __syncwarp();
#pragma unroll
        for (int i = 0; i < SIMT_VMAX; ++i) {
            const uint32_t e = l + 16 * i;
            if (e < a.vdim) {
                float o = acc[i] * r;
                for (int j = 0; j < SKT; ++j) o = fmaf(ps[qi * SKT + j], vs[j * a.vdim + e], o);
                acc[i] = o;
            }
        }
        __syncwarp();
    }
    if (t0 + qi < a.tokens) {
        const float g = (a.gate ? 1.0f / (1.0f + expf(-a.gate[(size_t)(t0 + qi) * a.ldg + h])) : 1.0f) * a.out_scale / lsum;
#pragma unroll
        for (int i = 0; i < SIMT_VMAX; ++i) {
            const uint32_t e = l + 16 * i;
            if (e < a.vdim) elem_store((T *)a.out + (size_t)(t0 + qi) * a.ldo + h * a.vdim + e, acc[i] * g);
        }
    }
}

// ---- tcgen05 -----------------------------------------------------------------------------------------------------------
constexpr uint32_t FW_WAIT = 1u << 22, BLK = 128 * 64 * 2;  // one [128][64] bf16 block, 16 KB
constexpr float SLACK = 8.0f;                               // in powers of two

struct WinMaps {
    CUtensorMap k, kr, v;
};

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// hi + lo = p: hi is p cut to 8 significant bits with rounding, lo the rest
__device__ __forceinline__ void split_bf16(float p0, float p1, uint32_t &hi, uint32_t &lo) {
    hi = bf16_pack(p0, p1);
    lo = bf16_pack(p0 - bf16_lo(hi), p1 - bf16_hi(hi));
}

// The exponential of four softcapped scores, in powers of two: with u = s * c2 (c2 = 2 log2(e) scale / cap) it is
// 2^(capl (1 - 2 / (1 + 2^u))), capl = cap log2(e). One reciprocal serves all four; past u = 29 the tanh is 1 in f32.
__device__ __forceinline__ void capped_exp4(float s[4], float c2, float capl) {
    float a[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) a[i] = 1.0f + ex2(fminf(s[i] * c2, 29.0f));
    const float p01 = a[0] * a[1], p23 = a[2] * a[3];
    float r;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(p01 * p23));
    const float r01 = r * p23, r23 = r * p01, m = -2.0f * capl;
    s[0] = ex2(fmaf(m, r01 * a[1], capl));
    s[1] = ex2(fmaf(m, r01 * a[0], capl));
    s[2] = ex2(fmaf(m, r23 * a[3], capl));
    s[3] = ex2(fmaf(m, r23 * a[2], capl));
}
constexpr float CAP_MAX = 64.0f;  // e^cap times the number of keys stays inside f32 up to here

// NU, NR: 64-column blocks of a key's own and its shared part (0: none); NV: of the values
template <int NU, int NR, int NV>
struct WinShape {
    static constexpr uint32_t NQ = NU + NR;
    static constexpr uint32_t KBUF = NQ <= 3 ? 2 : 1;  // K tiles in flight
    static constexpr size_t SMEM = (size_t)(NQ + KBUF * NQ + 2 * NV) * BLK + 1024;
};

template <int NU, int NR, int NV, bool CAP>
__global__ void __launch_bounds__(288, 1) window_tc_kernel(const __grid_constant__ WinMaps maps, WindowAttn a, uint32_t *status) {
    constexpr uint32_t NQ = NU + NR, KBUF = WinShape<NU, NR, NV>::KBUF;
    extern __shared__ __align__(1024) uint8_t smem_raw[];
    uint8_t *smem = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    uint8_t *qt = smem;
    auto KB = [&](uint32_t j) { return smem + (NQ + (KBUF == 2 ? (j & 1) : 0u) * NQ) * BLK; };
    auto VB = [&](uint32_t j) { return smem + (NQ + KBUF * NQ + (j & 1) * NV) * BLK; };
    __shared__ uint64_t bar_s[2], bar_k[2], bar_v[2], bar_o;
    __shared__ uint32_t tmem_base_s, abort_s;
    __shared__ float pair_max[2][128];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const uint32_t h = blockIdx.y, q0 = blockIdx.x * 128, nq = min(128u, a.tokens - q0), dq = a.dim + a.rot;
    const uint32_t qfirst = a.pos0 + q0, qlast = qfirst + nq - 1;
    // key tiles count from key0; the first visible position of the first query opens the sweep
    const uint32_t lo = max(a.key0, qfirst + 1 > a.window ? qfirst + 1 - a.window : 0u);
    const uint32_t jbeg = (lo - a.key0) / 128, nkt = (qlast - a.key0) / 128 + 1 - jbeg, kvh = h / (a.heads / a.kv_heads);
    auto tile_row = [&](uint32_t j) { return (int)(a.ring ? (a.key0 + (jbeg + j) * 128) % a.ring : (jbeg + j) * 128); };

    if (tid == 256) {  // the issuing thread, which asks for the first tiles before the block meets
        for (int i = 0; i < 2; ++i) {
            mbar_init(&bar_s[i], 1);
            mbar_init(&bar_k[i], 1);
            mbar_init(&bar_v[i], 1);
        }
        mbar_init(&bar_o, 1);
        abort_s = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {  // tensor memory: S at 0 and 128, O at 256, P hi at 384, P lo at 448
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base_s)), "r"(512u) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    pdl_wait();
    pdl_launch();
    uint32_t inflight = 0;  // issuing thread: bit b = a K copy into buffer b, bit 2 + b = a V copy, not yet waited for
    auto fetch_k = [&](uint32_t j) {
        const uint32_t b = KBUF == 2 ? (j & 1) : 0u;
        const int row = tile_row(j);
        mbar_expect_tx(&bar_k[b], NQ * BLK);
#pragma unroll
        for (int i = 0; i < NU; ++i) tma_load_3d(KB(j) + i * BLK, &maps.k, i * 64, (int)kvh, row, &bar_k[b]);
#pragma unroll
        for (int i = 0; i < NR; ++i) tma_load_2d(KB(j) + (NU + i) * BLK, &maps.kr, i * 64, row, &bar_k[b]);
        inflight |= 1u << b;
    };
    auto fetch_v = [&](uint32_t j) {
        mbar_expect_tx(&bar_v[j & 1], NV * BLK);
#pragma unroll
        for (int i = 0; i < NV; ++i) tma_load_3d(VB(j) + i * BLK, &maps.v, i * 64, (int)kvh, tile_row(j), &bar_v[j & 1]);
        inflight |= 4u << (j & 1);
    };
    if (tid == 256) {
        fetch_k(0);
        fetch_v(0);
        if (KBUF == 2 && nkt > 1) fetch_k(1);
    }
    // Q tile: rotated, rounded to bf16, swizzled K-major; rows past the last query and columns past the sizes are zeros
    const uint32_t half = a.rot_dims / 2;
    const bool qvec = ((a.ldq | dq | a.dim) & 3) == 0, rvec = (half & 7) == 0;
    const uint32_t own_rot = NR == 0 ? a.rot_dims : 0u;  // rotated columns of the own part
    for (uint32_t i = tid; i < 128 * NQ * 8; i += 288) {
        const uint32_t r = i / (NQ * 8), c = i - r * (NQ * 8), blk = c >> 3, c8 = (c & 7) * 8;
        uint32_t w[4] = {0, 0, 0, 0};
        if (r < nq) {
            const float *q = a.q + (size_t)(q0 + r) * a.ldq + h * dq;
            const uint32_t p = qfirst + r;
            const float *ct = a.cos_t + (size_t)p * half, *st = a.sin_t + (size_t)p * half;
            float v[8];
            if (qvec && blk < NU && blk * 64 + c8 >= own_rot && blk * 64 + c8 + 8 <= a.dim) {
                const float4 x = *reinterpret_cast<const float4 *>(q + blk * 64 + c8), y = *reinterpret_cast<const float4 *>(q + blk * 64 + c8 + 4);
                v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
                v[4] = y.x; v[5] = y.y; v[6] = y.z; v[7] = y.w;
            } else if (qvec && rvec && (blk >= NU || NR == 0) && (blk - (NR ? NU : 0)) * 64 + c8 + 8 <= a.rot_dims) {
                // eight neighbours of one half of the pairs
                const uint32_t e0 = (blk - (NR ? NU : 0)) * 64 + c8, f0 = e0 < half ? e0 : e0 - half;
                const float *own = q + (NR ? a.dim : 0) + e0, *other = e0 < half ? own + half : own - half;
                const float sign = e0 < half ? -1.0f : 1.0f;
#pragma unroll
                for (int u = 0; u < 8; u += 4) {
                    const float4 x = *reinterpret_cast<const float4 *>(own + u), y = *reinterpret_cast<const float4 *>(other + u);
                    const float4 cc = *reinterpret_cast<const float4 *>(ct + f0 + u), ss = *reinterpret_cast<const float4 *>(st + f0 + u);
                    v[u] = fmaf(sign * y.x, ss.x, x.x * cc.x);
                    v[u + 1] = fmaf(sign * y.y, ss.y, x.y * cc.y);
                    v[u + 2] = fmaf(sign * y.z, ss.z, x.z * cc.z);
                    v[u + 3] = fmaf(sign * y.w, ss.w, x.w * cc.w);
                }
            } else
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                const uint32_t col = (blk < NU ? blk : blk - NU) * 64 + c8 + e;
                if (NR == 0) v[e] = col < a.dim ? rotated(q, col, a.rot_dims, ct, st) : 0.0f;
                else if (blk < NU) v[e] = col < a.dim ? q[col] : 0.0f;
                else v[e] = col < a.rot ? rotated(q + a.dim, col, a.rot_dims, ct, st) : 0.0f;
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) w[e] = bf16_pack(v[2 * e], v[2 * e + 1]);
        }
        *reinterpret_cast<uint4 *>(qt + blk * BLK + (r >> 3) * 1024 + (r & 7) * 128 + (((c8 >> 3) ^ (r & 7)) << 4)) = make_uint4(w[0], w[1], w[2], w[3]);
    }
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = tmem_base_s, tmem_o = tmem + 256, tmem_p = tmem + 384;
    volatile uint32_t *abort_flag = &abort_s;
    auto wait = [&](uint64_t *bar, uint32_t parity) -> bool {
        for (uint32_t it = 0; it < FW_WAIT; ++it) {
            if (tc_mbar_try(bar, parity)) return true;
            if (*abort_flag) return false;
        }
        atomicExch(status, 7u);
        *abort_flag = 1;
        return false;
    };
    constexpr uint32_t idesc_s = tc_idesc_bf16(128, 128), idesc_o = tc_idesc_bf16(128, NV * 64) | (1u << 16);  // V: an MN-major B operand
    auto issue_s = [&](uint32_t j) {
        const uint32_t q = smem_u32(qt), k = smem_u32(KB(j));
#pragma unroll
        for (uint32_t b = 0; b < NQ; ++b)
#pragma unroll
            for (uint32_t ks = 0; ks < 4; ++ks)
                tc_mma(tmem + 128 * (j & 1), tc_desc_kmajor(q + b * BLK + ks * 32), tc_desc_kmajor(k + b * BLK + ks * 32), idesc_s, (b > 0 || ks > 0) ? 1u : 0u);
        tc_commit(&bar_s[j & 1]);
    };
    const bool issuer = tid == 256, softmax = tid < 256;
    const uint32_t row = (warp & 3) * 32 + lane, cgrp = (warp >> 2) & 1, c0 = cgrp * 64, trow = ((warp & 3) * 32u) << 16;
    const uint32_t qpos = qfirst + row;
    const float sl = a.scale * LOG2E, c2 = CAP ? 2.0f * sl / a.softcap : 0.0f, capl = a.softcap * LOG2E;
    float m = -INFINITY, l = 0.0f;  // reference value and row sum, in powers of two of the scaled score
    uint32_t phs = 0, phk = 0, phv = 0, ph_o = 0;  // bit b: parity of buffer b's barrier
    bool ok = true;
    auto wait_k = [&](uint32_t j) -> bool {
        const uint32_t b = KBUF == 2 ? (j & 1) : 0u;
        const bool r = wait(&bar_k[b], (phk >> b) & 1);
        phk ^= 1u << b;
        if (r) inflight &= ~(1u << b);
        return r;
    };
    auto wait_v = [&](uint32_t j) -> bool {
        const uint32_t b = j & 1;
        const bool r = wait(&bar_v[b], (phv >> b) & 1);
        phv ^= 1u << b;
        if (r) inflight &= ~(4u << b);
        return r;
    };
    if (issuer) {
        if (wait_k(0)) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            issue_s(0);
        }
    }
    for (uint32_t j = 0; j < nkt && ok; ++j) {
        if (KBUF == 2 && issuer && j + 1 < nkt && wait_k(j + 1)) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            issue_s(j + 1);
        }
        ok = wait(&bar_s[j & 1], (phs >> (j & 1)) & 1);
        phs ^= 1u << (j & 1);
        ok = __all_sync(0xffffffffu, ok);
        if (ok && issuer) {  // S of tile j is formed: its K buffer is free
            if (KBUF == 2) {
                if (j + 2 < nkt) fetch_k(j + 2);
            } else if (j + 1 < nkt) {
                fetch_k(j + 1);
            }
        }
        uint32_t hi[32], lo_[32];
        float rescale = 1.0f;
        bool move = false;
        if (ok && softmax) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t ts = tmem + 128 * (j & 1) + trow + c0;
            const uint32_t k0 = a.key0 + (jbeg + j) * 128;  // position of the tile's first key
            const bool free_tile = k0 + 127 <= qfirst && k0 + a.window > qfirst + 127;
            // a key of column c is visible when lob <= c <= hib
            const int hib = (int)qpos - (int)(k0 + c0), lob = hib - (int)a.window + 1;
            if constexpr (CAP) {
#pragma unroll
                for (int cc = 0; cc < 2; ++cc) {
                    uint32_t v[32];
                    tc_ld32(ts + 32 * cc, v);
#pragma unroll
                    for (int i = 0; i < 32; i += 4) {
                        float p[4];
#pragma unroll
                        for (int e = 0; e < 4; ++e) p[e] = __uint_as_float(v[i + e]);
                        capped_exp4(p, c2, capl);
                        if (!free_tile)
#pragma unroll
                            for (int e = 0; e < 4; ++e)
                                if (32 * cc + i + e > hib || 32 * cc + i + e < lob) p[e] = 0.0f;
                        l += (p[0] + p[1]) + (p[2] + p[3]);
                        split_bf16(p[0], p[1], hi[16 * cc + i / 2], lo_[16 * cc + i / 2]);
                        split_bf16(p[2], p[3], hi[16 * cc + i / 2 + 1], lo_[16 * cc + i / 2 + 1]);
                    }
                }
            } else {
                float tmax = -INFINITY;
#pragma unroll
                for (int cc = 0; cc < 2; ++cc) {
                    uint32_t v[32];
                    tc_ld32(ts + 32 * cc, v);
                    if (free_tile) {
#pragma unroll
                        for (int i = 0; i < 32; ++i) tmax = fmaxf(tmax, __uint_as_float(v[i]) * sl);
                    } else {
#pragma unroll
                        for (int i = 0; i < 32; ++i)
                            if (32 * cc + i <= hib && 32 * cc + i >= lob) tmax = fmaxf(tmax, __uint_as_float(v[i]) * sl);
                    }
                }
                pair_max[cgrp][row] = tmax;
                asm volatile("bar.sync %0, %1;" ::"r"(1 + (warp & 3)), "r"(64) : "memory");  // the two warps that share these rows
                tmax = fmaxf(pair_max[0][row], pair_max[1][row]);
                if (tmax > m + SLACK || (m == -INFINITY && tmax != -INFINITY)) {
                    move = m != -INFINITY;
                    rescale = move ? ex2(m - tmax) : 1.0f;
                    l *= rescale;
                    m = tmax;
                }
                const float mneg = m == -INFINITY ? 0.0f : -m;
#pragma unroll
                for (int cc = 0; cc < 2; ++cc) {
                    uint32_t v[32];
                    tc_ld32(ts + 32 * cc, v);
#pragma unroll
                    for (int i = 0; i < 32; i += 2) {
                        float p0 = ex2(fmaf(__uint_as_float(v[i]), sl, mneg)), p1 = ex2(fmaf(__uint_as_float(v[i + 1]), sl, mneg));
                        if (!free_tile) {
                            const int c = 32 * cc + i;
                            if (c > hib || c < lob) p0 = 0.0f;
                            if (c + 1 > hib || c + 1 < lob) p1 = 0.0f;
                        }
                        l += p0 + p1;
                        split_bf16(p0, p1, hi[16 * cc + i / 2], lo_[16 * cc + i / 2]);
                    }
                }
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
        }
        if (ok && j > 0) {  // P and the other V buffer are free once P V of tile j - 1 has finished
            ok = wait(&bar_o, ph_o);
            ph_o ^= 1;
            ok = __all_sync(0xffffffffu, ok);
        }
        if (ok && issuer && j + 1 < nkt) fetch_v(j + 1);
        if (ok && softmax) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            if (!CAP && j > 0 && __any_sync(0xffffffffu, move)) {
                // a row's reference moved: what O holds for it was accumulated against the old one; each thread of the pair
                // scales its half of the value columns
#pragma unroll 1
                for (uint32_t c = cgrp * (NV * 32); c < (cgrp + 1) * (NV * 32); c += 32) {
                    uint32_t v[32];
                    tc_ld32(tmem_o + trow + c, v);
#pragma unroll
                    for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * rescale);
                    tc_st32(tmem_o + trow + c, v);
                }
            }
            tc_st32(tmem_p + trow + c0 / 2, hi);
            tc_st32(tmem_p + 64 + trow + c0 / 2, lo_);
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
        }
        ok = __syncthreads_and(ok);  // P of tile j is complete; every read of S of tile j is done
        if (!ok) break;
        if (issuer) {  // O += P_hi V + P_lo V over the tile's 128 keys, 16 per instruction
            if (wait_v(j)) {
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll
                for (uint32_t ks = 0; ks < 8; ++ks) {
                    const uint64_t dv = tc_desc_mnmajor(smem_u32(VB(j)) + ks * 2048);
                    tc_mma_ta(tmem_o, tmem_p + 8 * ks, dv, idesc_o, (j > 0 || ks > 0) ? 1u : 0u);
                    tc_mma_ta(tmem_o, tmem_p + 64 + 8 * ks, dv, idesc_o, 1u);
                }
                tc_commit(&bar_o);
                if (KBUF == 1 && j + 1 < nkt && wait_k(j + 1)) {
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    issue_s(j + 1);
                }
            }
        }
    }
    if (ok) {
        ok = wait(&bar_o, ph_o);
        ok = __all_sync(0xffffffffu, ok);
    }
    ok = __syncthreads_and(ok);
    if (ok) {
        if (softmax) pair_max[cgrp][row] = l;
        __syncthreads();
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        if (softmax) {
            const float total = pair_max[0][row] + pair_max[1][row];
            float g = 0.0f;
            if (row < nq) g = (a.gate ? 1.0f / (1.0f + expf(-a.gate[(size_t)(q0 + row) * a.ldg + h])) : 1.0f) * a.out_scale / total;
            __nv_bfloat16 *dst = (__nv_bfloat16 *)a.out + (size_t)(q0 + row) * a.ldo + h * a.vdim;
            const bool vec = ((a.ldo | a.vdim) & 7) == 0;
#pragma unroll 1
            for (uint32_t c = cgrp * (NV * 32); c < (cgrp + 1) * (NV * 32); c += 32) {
                uint32_t v[32];
                tc_ld32(tmem_o + trow + c, v);
                if (row < nq) {
#pragma unroll
                    for (int e = 0; e < 32; e += 8) {
                        if (vec && c + e + 8 <= a.vdim) {
                            uint32_t w[4];
#pragma unroll
                            for (int i = 0; i < 4; ++i) w[i] = bf16_pack(__uint_as_float(v[e + 2 * i]) * g, __uint_as_float(v[e + 2 * i + 1]) * g);
                            *reinterpret_cast<uint4 *>(dst + c + e) = make_uint4(w[0], w[1], w[2], w[3]);
                        } else {
#pragma unroll
                            for (int i = 0; i < 8; ++i)
                                if (c + e + i < a.vdim) dst[c + e + i] = __float2bfloat16_rn(__uint_as_float(v[e + i]) * g);
                        }
                    }
                }
            }
        }
    } else if (issuer) {  // a wait gave up: let the copies in flight land before the CTA exits
        for (int b = 0; b < 2; ++b) {
            if (inflight & (1u << b))
                for (uint32_t it = 0; it < FW_WAIT && !tc_mbar_try(&bar_k[b], (phk >> b) & 1); ++it) {}
            if (inflight & (4u << b))
                for (uint32_t it = 0; it < FW_WAIT && !tc_mbar_try(&bar_v[b], (phv >> b) & 1); ++it) {}
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
    }
}

template <int NU, int NR, int NV, bool CAP>
int32_t launch_window_tc(brasa_cmd *cmd, const WindowAttn &a) {
    brasa_ctx *ctx = cmd->ctx;
    WinMaps maps;
    // (columns between a head's size and its step are never read: they lie outside the map, or the query tile has zeros there
    // and the output leaves them out)
    const uint64_t rows = a.ring ? a.ring : a.keys;
    const uint64_t kd[3] = {(a.dim + 7) / 8 * 8, a.kv_heads, rows}, kst[2] = {(uint64_t)a.kstep * 2, (uint64_t)a.ldk * 2};
    const uint64_t vd[3] = {(a.vdim + 7) / 8 * 8, a.kv_heads, rows}, vst[2] = {(uint64_t)a.vstep * 2, (uint64_t)a.ldv * 2};
    const uint32_t box3[3] = {64, 1, 128}, box2[2] = {64, 128};
    BRASA_TRY(brasa_tmap_bf16(ctx, &maps.k, 3, a.k, kd, kst, box3));
    BRASA_TRY(brasa_tmap_bf16(ctx, &maps.v, 3, a.v, vd, vst, box3));
    maps.kr = maps.k;
    if (NR) {
        const uint64_t rd[2] = {a.rot, rows}, rst[1] = {(uint64_t)a.ldr * 2};
        BRASA_TRY(brasa_tmap_bf16(ctx, &maps.kr, 2, a.kr, rd, rst, box2));
    }
    const size_t smem = WinShape<NU, NR, NV>::SMEM;
    BRASA_TRY(brasa_smem_optin(ctx, (const void *)window_tc_kernel<NU, NR, NV, CAP>, smem));
    BRASA_CUDA(ctx, brasa_launch_dependent(ctx, window_tc_kernel<NU, NR, NV, CAP>, dim3((a.tokens + 127) / 128, a.heads), dim3(288), smem, maps, a, ctx->status));
    return brasa_post_launch(cmd, "window_tc");
}

template <int NU, int NV>
int32_t launch_window_own(brasa_cmd *cmd, const WindowAttn &a) {
    return a.softcap > 0.0f ? launch_window_tc<NU, 0, NV, true>(cmd, a) : launch_window_tc<NU, 0, NV, false>(cmd, a);
}

template <typename T>
int32_t launch_window_simt(brasa_cmd *cmd, const WindowAttn &a) {
    brasa_ctx *ctx = cmd->ctx;
    const uint32_t dq = a.dim + a.rot;
    const size_t smem = ((size_t)SQ * dq + (size_t)SKT * (dq + 1) + (size_t)SKT * a.vdim + SQ * SKT) * 4;
    BRASA_REQUIRE(ctx, a.vdim <= 16 * SIMT_VMAX && smem + 1024 <= ctx->smem_optin, "window attention: head sizes too large");
    BRASA_TRY(brasa_smem_optin(ctx, (const void *)window_simt_kernel<T>, smem));
    BRASA_CUDA(ctx, brasa_launch_dependent(ctx, window_simt_kernel<T>, dim3((a.tokens + SQ - 1) / SQ, a.heads), dim3(256), smem, a));
    return brasa_post_launch(cmd, "window_simt");
}

}  // namespace

int32_t brasa_window_attention_launch(brasa_cmd *cmd, const WindowAttn &a, bool f32) {
    BRASA_REQUIRE(cmd->ctx, a.tokens > 0 && a.heads > 0 && a.window > 0 && a.key0 <= a.pos0 && a.key0 + a.keys == a.pos0 + a.tokens && (a.rot == 0 || a.rot_dims <= a.rot) &&
                                a.rot_dims % 2 == 0,
                  "window attention: bad range or sizes");
    BRASA_REQUIRE(cmd->ctx, a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.kstep >= a.dim && a.vstep >= a.vdim && (a.rot > 0 || a.rot_dims <= a.dim) && a.softcap >= 0.0f,
                  "window attention: bad heads or steps");
    BRASA_REQUIRE(cmd->ctx, !a.ring || (a.ring % 128 == 0 && a.key0 % 128 == 0), "window attention: a ring and its first key are multiples of 128");
    if (f32) return launch_window_simt<float>(cmd, a);
    const uint32_t nu = (a.dim + 63) / 64, nr = (a.rot + 63) / 64, nv = (a.vdim + 63) / 64;
    if (((a.kstep | a.vstep | a.ldk | a.ldv | a.ldr) & 7) == 0) {
        if (nr == 1 && a.softcap == 0.0f) {
            if (nu == 1 && nv == 1) return launch_window_tc<1, 1, 1, false>(cmd, a);
            if (nu == 1 && nv == 2) return launch_window_tc<1, 1, 2, false>(cmd, a);
            if (nu == 2 && nv == 1) return launch_window_tc<2, 1, 1, false>(cmd, a);
            if (nu == 2 && nv == 2) return launch_window_tc<2, 1, 2, false>(cmd, a);
            if (nu == 3 && nv == 1) return launch_window_tc<3, 1, 1, false>(cmd, a);
            if (nu == 3 && nv == 2) return launch_window_tc<3, 1, 2, false>(cmd, a);
        }
        if (nr == 0 && a.softcap <= CAP_MAX) {
            if (nu == 1 && nv == 1) return launch_window_own<1, 1>(cmd, a);
            if (nu == 1 && nv == 2) return launch_window_own<1, 2>(cmd, a);
            if (nu == 2 && nv == 1) return launch_window_own<2, 1>(cmd, a);
            if (nu == 2 && nv == 2) return launch_window_own<2, 2>(cmd, a);
            if (nu == 3 && nv == 1) return launch_window_own<3, 1>(cmd, a);
            if (nu == 3 && nv == 2) return launch_window_own<3, 2>(cmd, a);
        }
    }
    return launch_window_simt<__nv_bfloat16>(cmd, a);
}

extern "C" int32_t brasa_k_window_attention(brasa_cmd *cmd, brasa_window_attn p, int32_t f32) {
    if (!cmd) return BRASA_EINVAL;
    brasa_ctx *ctx = cmd->ctx;
    BRASA_REQUIRE(ctx, p.tokens > 0 && p.heads > 0 && p.dim > 0 && p.vdim > 0 && p.window > 0 && p.key0 <= p.pos0 && p.kv_heads > 0 && p.heads % p.kv_heads == 0,
                  "window attention: empty shape");
    BRASA_REQUIRE(ctx, p.rot % 8 == 0 && p.rot_dims <= (p.rot ? p.rot : p.dim) && (p.key0 == 0 || p.key0 + p.window <= p.pos0 + 1),
                  "window attention: rot must be a multiple of 8 and every visible key present");
    const uint64_t keys = (uint64_t)p.pos0 + p.tokens - p.key0, e = f32 ? 4 : 2, last = (uint64_t)p.pos0 + p.tokens, rows = p.ring ? p.ring : keys;
    BRASA_REQUIRE(ctx, !p.ring || std::min<uint64_t>(p.window - 1, p.pos0) + p.tokens <= p.ring, "window attention: the ring is shorter than the window and the run");
    BRASA_REQUIRE(ctx, arg_fits(p.q, (uint64_t)p.tokens * p.heads * (p.dim + p.rot) * 4) && arg_fits(p.k, rows * p.kv_heads * p.dim * e) &&
                           arg_fits(p.v, rows * p.kv_heads * p.vdim * e) && (!p.rot || arg_fits(p.kr, rows * p.rot * e)) &&
                           (!p.gate.buf || arg_fits(p.gate, (uint64_t)p.tokens * p.heads * 4)) && arg_fits(p.out, (uint64_t)p.tokens * p.heads * p.vdim * e) &&
                           arg_fits(p.cos_t, last * (p.rot_dims / 2) * 4) && arg_fits(p.sin_t, last * (p.rot_dims / 2) * 4),
                  "window attention: a buffer is too small");
    for (const brasa_arg *a : {&p.k, &p.v, &p.kr, &p.out}) BRASA_REQUIRE(ctx, a->offset % 16 == 0, "window attention: misaligned buffer");
    WindowAttn a{};
    a.q = (const float *)arg_ptr(p.q);
    a.k = arg_ptr(p.k);
    a.v = arg_ptr(p.v);
    a.kr = arg_ptr(p.kr);
    a.cos_t = (const float *)arg_ptr(p.cos_t);
    a.sin_t = (const float *)arg_ptr(p.sin_t);
    a.gate = (const float *)arg_ptr(p.gate);
    a.out = arg_ptr(p.out);
    a.ldq = p.heads * (p.dim + p.rot);
    a.ldk = p.kv_heads * p.dim;
    a.ldv = p.kv_heads * p.vdim;
    a.ldo = p.heads * p.vdim;
    a.ldr = p.rot;
    a.ldg = p.heads;
    a.tokens = p.tokens; a.heads = p.heads; a.dim = p.dim; a.rot = p.rot; a.rot_dims = p.rot_dims; a.vdim = p.vdim;
    a.pos0 = p.pos0; a.key0 = p.key0; a.keys = (uint32_t)keys; a.window = p.window;
    a.scale = p.scale;
    a.kv_heads = p.kv_heads; a.kstep = p.dim; a.vstep = p.vdim;
    a.ring = p.ring;
    a.softcap = p.softcap;
    a.out_scale = p.out_scale;
    return brasa_window_attention_launch(cmd, a, f32 != 0);
}
