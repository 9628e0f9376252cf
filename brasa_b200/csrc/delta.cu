// Gated delta rule with one decay per key channel ("channel_delta"), a recurrent mixer. A head keeps a matrix S [dim][vdim] of
// what each key direction stands for. A token fades the rows of S by its decays g, reads what its key k finds there, moves that
// towards its value v by the fraction beta, and its query q reads the result:
//   F = diag(g) S_old,  u = beta (v - F^T k),  S_new = F + k u^T,  o = S_new^T q
// q, k and v come out of a short causal convolution and silu, q and k as unit vectors, g out of a softplus.
//
// Many tokens: delta_prep_kernel forms q, k, v, g and beta of every token side by side; delta_scan_kernel then walks the
// tokens with the state in registers. 16 lanes share a state column (each a slice of the key channels), and because
// S_new^T q = F^T q + u (k . q), both reductions of a token run together and a token costs one exchange between
// lanes. Everything is f32 FMA in the order of the tokens, so a sequence cut into portions gives the same bits.
// One token: delta_step_kernel does all of it, one block per head.
//
// Per-sequence state: S [heads][dim][vdim] and the convolution's inputs as a ring of `taps` rows, position p in row p % taps
// (one more row than needed, so that a step can store its own row while others still read the older ones). A sequence
// starts at position 0 by ignoring both.
#include <cuda_bf16.h>

#include "stack.h"
#include "tc_device.cuh"

using namespace brasa_dev;

namespace {

constexpr float UNIT_EPS = 1e-6f;

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

struct DeltaShape {
    uint32_t heads, kv_heads, dim, vdim, taps;
    uint32_t qk;  // kv_heads * dim
    uint32_t vd;  // heads * vdim
};

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

struct DeltaPrep {
    DeltaShape s;
    ConvView cv;
    const float *q, *k, *v, *b, *z;       // products [tokens][ld]
    uint32_t ldqk, ldv, ldb, ldz;
    const float *wq, *wk, *wv, *a_log;
    float *qn, *kn, *vn, *g, *beta, *kq;  // [tokens][qk], [qk], [vd], [heads * dim], [heads], [kv_heads]
};

// One warp per kv head (q and k), head (v) or head (g and beta) of a token.
__global__ void __launch_bounds__(256) delta_prep_kernel(DeltaPrep p) {
    pdl_wait();
    pdl_launch();
    const DeltaShape s = p.s;
    const uint32_t t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, items = s.kv_heads + 2 * s.heads;
    for (uint32_t it = blockIdx.y * 8 + warp; it < items; it += gridDim.y * 8) {
        if (it < s.kv_heads) {
            float q[8], k[8], qq = 0.0f, kk = 0.0f, kq = 0.0f;
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const uint32_t i = lane + 32 * j, c = it * s.dim + i;
                q[j] = k[j] = 0.0f;
                if (i < s.dim) {
                    q[j] = silu_f(conv_at(p.q, p.ldqk, c, p.wq, t, p.cv, c));
                    k[j] = silu_f(conv_at(p.k, p.ldqk, c, p.wk, t, p.cv, s.qk + c));
                }
                qq = fmaf(q[j], q[j], qq);
                kk = fmaf(k[j], k[j], kk);
            }
            qq = 1.0f / (sqrtf(warp_sum(qq) + UNIT_EPS) * sqrtf((float)s.dim));
            kk = 1.0f / sqrtf(warp_sum(kk) + UNIT_EPS);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const uint32_t i = lane + 32 * j;
                q[j] *= qq;
                k[j] *= kk;
                kq = fmaf(k[j], q[j], kq);
                if (i < s.dim) {
                    p.qn[(size_t)t * s.qk + it * s.dim + i] = q[j];
                    p.kn[(size_t)t * s.qk + it * s.dim + i] = k[j];
                }
            }
            kq = warp_sum(kq);
            if (lane == 0) p.kq[(size_t)t * s.kv_heads + it] = kq;
        } else if (it < s.kv_heads + s.heads) {
            const uint32_t h = it - s.kv_heads;
            for (uint32_t i = lane; i < s.vdim; i += 32) {
                const uint32_t c = h * s.vdim + i;
                p.vn[(size_t)t * s.vd + c] = silu_f(conv_at(p.v, p.ldv, c, p.wv, t, p.cv, 2 * s.qk + c));
            }
        } else {
            const uint32_t h = it - s.kv_heads - s.heads;
            const float a = expf(p.a_log[h]);
            for (uint32_t i = lane; i < s.dim; i += 32)
                p.g[(size_t)t * s.heads * s.dim + h * s.dim + i] = expf(-a * softplus_f(p.z[(size_t)t * p.ldz + h * s.dim + i]));
            if (lane == 0) p.beta[(size_t)t * s.heads + h] = sigmoid_f(p.b[(size_t)t * p.ldb + h]);
        }
    }
}

// The run's last inputs of the convolution into the ring.
__global__ void __launch_bounds__(256) delta_ring_kernel(DeltaShape s, const float *q, const float *k, const float *v, uint32_t ldqk, uint32_t ldv,
                                                         float *ring, uint32_t tokens, uint32_t pos0) {
    pdl_wait();
    pdl_launch();
    const uint32_t channels = 2 * s.qk + s.vd, ch = blockIdx.x * 256 + threadIdx.x;
    if (ch >= channels) return;
    const uint32_t n = min(tokens, s.taps);
    for (uint32_t t = tokens - n; t < tokens; ++t) {
        const float x = ch < s.qk ? q[(size_t)t * ldqk + ch] : (ch < 2 * s.qk ? k[(size_t)t * ldqk + ch - s.qk] : v[(size_t)t * ldv + ch - 2 * s.qk]);
        ring[(size_t)((pos0 + t) % s.taps) * channels + ch] = x;
    }
}

struct DeltaScan {
    DeltaShape s;
    const float *qn, *kn, *vn, *g, *beta, *kq;
    float *state;  // [heads][dim][vdim]
    float *o;      // [tokens][vd]
    uint32_t tokens;
    int fresh;     // the sequence starts here: the state is zero, whatever is stored
};

__device__ __forceinline__ void cp4(float *dst, const float *src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp16(float *dst, const float *src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

// Block: one head, 16 * CPT state columns; thread = (lane of 16, column pair). Lane l of a column owns rows
// 4 (l + 16 j) .. + 3, j < RPT / 4.
template <int RPT, int CPT>
__global__ void __launch_bounds__(256) delta_scan_kernel(DeltaScan p) {
    constexpr int D = 16 * RPT, CB = 16 * CPT, SCAN_TOK = RPT > 8 ? 4 : 8;  // SCAN_TOK: tokens per stage
    __shared__ __align__(16) float sq[2][SCAN_TOK][D], sk[2][SCAN_TOK][D], sg[2][SCAN_TOK][D], sv[2][SCAN_TOK][CB], sc[2][SCAN_TOK][2], so[SCAN_TOK][CB];
    const DeltaShape s = p.s;
    const uint32_t h = blockIdx.x, kh = h / (s.heads / s.kv_heads), c0 = blockIdx.y * CB;
    const int tid = threadIdx.x, l = tid & 15, cp = tid >> 4;
    const uint32_t col = c0 + cp * CPT;
    // rows past dim stay zero in every stage: zero k and q leave the padded rows of the state at zero
    for (int i = tid; i < 2 * SCAN_TOK * D; i += 256) {
        (&sq[0][0][0])[i] = 0.0f;
        (&sk[0][0][0])[i] = 0.0f;
        (&sg[0][0][0])[i] = 0.0f;
    }
    for (int i = tid; i < 2 * SCAN_TOK * CB; i += 256) (&sv[0][0][0])[i] = 0.0f;
    __syncthreads();
    pdl_wait();
    pdl_launch();
    float S[RPT][CPT];
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
        const uint32_t row = 4 * (l + 16 * (r >> 2)) + (r & 3);
#pragma unroll
        for (int c = 0; c < CPT; ++c)
            S[r][c] = (!p.fresh && row < s.dim && col + c < s.vdim) ? p.state[((size_t)h * s.dim + row) * s.vdim + col + c] : 0.0f;
    }
    const uint32_t ncol = min((uint32_t)CB, s.vdim - c0);
    const bool vec = (s.dim & 3) == 0;
    auto fetch = [&](uint32_t t0, int b) {
        const uint32_t n = min((uint32_t)SCAN_TOK, p.tokens - t0);
        if (vec) {
            const uint32_t d4 = s.dim / 4;
            for (uint32_t i = tid; i < n * d4; i += 256) {
                const uint32_t t = i / d4, e = (i - t * d4) * 4;
                cp16(&sq[b][t][e], p.qn + (size_t)(t0 + t) * s.qk + kh * s.dim + e);
                cp16(&sk[b][t][e], p.kn + (size_t)(t0 + t) * s.qk + kh * s.dim + e);
                cp16(&sg[b][t][e], p.g + ((size_t)(t0 + t) * s.heads + h) * s.dim + e);
            }
        } else {
            for (uint32_t i = tid; i < n * s.dim; i += 256) {
                const uint32_t t = i / s.dim, e = i - t * s.dim;
                cp4(&sq[b][t][e], p.qn + (size_t)(t0 + t) * s.qk + kh * s.dim + e);
                cp4(&sk[b][t][e], p.kn + (size_t)(t0 + t) * s.qk + kh * s.dim + e);
                cp4(&sg[b][t][e], p.g + ((size_t)(t0 + t) * s.heads + h) * s.dim + e);
            }
        }
        for (uint32_t i = tid; i < n * ncol; i += 256) {
            const uint32_t t = i / ncol, e = i - t * ncol;
            cp4(&sv[b][t][e], p.vn + (size_t)(t0 + t) * s.vd + h * s.vdim + c0 + e);
        }
        for (uint32_t t = tid; t < n; t += 256) {
            cp4(&sc[b][t][0], p.beta + (size_t)(t0 + t) * s.heads + h);
            cp4(&sc[b][t][1], p.kq + (size_t)(t0 + t) * s.kv_heads + kh);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0, 0);
    for (uint32_t t0 = 0, b = 0; t0 < p.tokens; t0 += SCAN_TOK, b ^= 1) {
        if (t0 + SCAN_TOK < p.tokens) {
            fetch(t0 + SCAN_TOK, b ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const uint32_t n = min((uint32_t)SCAN_TOK, p.tokens - t0);
        for (uint32_t t = 0; t < n; ++t) {
            float k[RPT], rk[CPT] = {}, rq[CPT] = {};
#pragma unroll
            for (int j = 0; j < RPT / 4; ++j) {
                const int e = 4 * (l + 16 * j);
                const float4 k4 = *reinterpret_cast<const float4 *>(&sk[b][t][e]), q4 = *reinterpret_cast<const float4 *>(&sq[b][t][e]),
                             g4 = *reinterpret_cast<const float4 *>(&sg[b][t][e]);
                const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w}, gg[4] = {g4.x, g4.y, g4.z, g4.w};
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    k[4 * j + i] = kk[i];
#pragma unroll
                    for (int c = 0; c < CPT; ++c) {
                        S[4 * j + i][c] *= gg[i];
                        rk[c] = fmaf(kk[i], S[4 * j + i][c], rk[c]);
                        rq[c] = fmaf(qq[i], S[4 * j + i][c], rq[c]);
                    }
                }
            }
#pragma unroll
            for (int o = 8; o > 0; o >>= 1)
#pragma unroll
                for (int c = 0; c < CPT; ++c) {
                    rk[c] += __shfl_xor_sync(0xffffffffu, rk[c], o);
                    rq[c] += __shfl_xor_sync(0xffffffffu, rq[c], o);
                }
            const float beta = sc[b][t][0], kq = sc[b][t][1];
#pragma unroll
            for (int c = 0; c < CPT; ++c) {
                const float u = beta * (sv[b][t][cp * CPT + c] - rk[c]);
#pragma unroll
                for (int r = 0; r < RPT; ++r) S[r][c] = fmaf(k[r], u, S[r][c]);
                if (l == 0) so[t][cp * CPT + c] = fmaf(u, kq, rq[c]);
            }
        }
        __syncthreads();
        for (uint32_t i = tid; i < n * ncol; i += 256) {
            const uint32_t t = i / ncol, e = i - t * ncol;
            p.o[(size_t)(t0 + t) * s.vd + h * s.vdim + c0 + e] = so[t][e];
        }
    }
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
        const uint32_t row = 4 * (l + 16 * (r >> 2)) + (r & 3);
#pragma unroll
        for (int c = 0; c < CPT; ++c)
            if (row < s.dim && col + c < s.vdim) p.state[((size_t)h * s.dim + row) * s.vdim + col + c] = S[r][c];
    }
}

// o / rms(o) * w * sigmoid(gate), per head; one warp per (token, head)
template <typename T>
__global__ void __launch_bounds__(256) delta_out_kernel(const float *o, const float *gate, uint32_t ldg, const float *w, T *out, uint32_t ldo, uint32_t heads,
                                                        uint32_t vdim, uint32_t tokens, float eps) {
    pdl_wait();
    pdl_launch();
    const uint32_t i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (i >= tokens * heads) return;
    const uint32_t t = i / heads, h = i - t * heads;
    const float *x = o + (size_t)t * heads * vdim + h * vdim;
    float ss = 0.0f;
    for (uint32_t e = lane; e < vdim; e += 32) ss = fmaf(x[e], x[e], ss);
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + eps);
    for (uint32_t e = lane; e < vdim; e += 32)
        elem_store(out + (size_t)t * ldo + h * vdim + e, x[e] * inv * w[e] * sigmoid_f(gate[(size_t)t * ldg + h * vdim + e]));
}

// ---- one token ---------------------------------------------------------------------------------------------------------
struct DeltaStep {
    DeltaShape s;
    const float *q, *k, *v, *b, *a1, *g1;        // products of this token
    const float *wq, *wk, *wv, *a_log, *dt_bias, *norm;
    const uint16_t *wa2, *wg2;
    uint32_t ra, rg, lda2, ldg2;
    float *ring, *state, *out;
    const uint32_t *pos;
    float eps;
};
constexpr int STEP_THREADS = 512, STEP_R = 8, STEP_C = 4;  // state kept in registers up to 128 x 128

__device__ __forceinline__ float row_dot(const uint16_t *w, const float *x, uint32_t n, uint32_t lane) {
    float s = 0.0f;
    for (uint32_t c = lane * 8; c < n; c += 256) {
        const uint4 q = *reinterpret_cast<const uint4 *>(w + c);
        s = fmaf(bf16_lo(q.x), x[c], s);
        s = fmaf(bf16_hi(q.x), x[c + 1], s);
        s = fmaf(bf16_lo(q.y), x[c + 2], s);
        s = fmaf(bf16_hi(q.y), x[c + 3], s);
        s = fmaf(bf16_lo(q.z), x[c + 4], s);
        s = fmaf(bf16_hi(q.z), x[c + 5], s);
        s = fmaf(bf16_lo(q.w), x[c + 6], s);
        s = fmaf(bf16_hi(q.w), x[c + 7], s);
    }
    return warp_sum(s);
}

// Block = head. Warp w owns state rows w, w + 16, ..; lanes run along the columns.
template <bool KEEP>
__global__ void __launch_bounds__(STEP_THREADS, 1) delta_step_kernel(DeltaStep p) {
    extern __shared__ __align__(16) float sm[];
    const DeltaShape s = p.s;
    const uint32_t h = blockIdx.x, kh = h / (s.heads / s.kv_heads), ra8 = (p.ra + 7) / 8 * 8, rg8 = (p.rg + 7) / 8 * 8;
    float *sq = sm, *sk = sq + s.dim, *sg = sk + s.dim, *sv = sg + s.dim, *gate = sv + s.vdim, *o = gate + s.vdim, *rk = o + s.vdim,
          *rq = rk + 16 * s.vdim, *red = rq + 16 * s.vdim, *a1 = red + 8 + ((0u - (3 * s.dim + 35 * s.vdim)) & 3u), *g1 = a1 + ra8;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    float *S = p.state + (size_t)h * s.dim * s.vdim;
    float keep[STEP_R][STEP_C];
    if (KEEP) {  // no kernel that may still be running writes the state
#pragma unroll
        for (int r = 0; r < STEP_R; ++r)
#pragma unroll
            for (int c = 0; c < STEP_C; ++c) {
                const uint32_t row = warp + 16 * r, col = lane + 32 * c;
                keep[r][c] = (row < s.dim && col < s.vdim) ? S[(size_t)row * s.vdim + col] : 0.0f;
            }
    }
    pdl_wait();
    pdl_launch();
    const uint32_t pos = *p.pos;
    const bool fresh = pos == 0;
    const ConvView cv{p.ring, 2 * s.qk + s.vd, s.taps, pos};
    for (uint32_t i = tid; i < ra8; i += STEP_THREADS) a1[i] = i < p.ra ? p.a1[i] : 0.0f;
    for (uint32_t i = tid; i < rg8; i += STEP_THREADS) g1[i] = i < p.rg ? p.g1[i] : 0.0f;
    for (uint32_t i = tid; i < 2 * s.dim + s.vdim; i += STEP_THREADS) {
        if (i < s.dim) sq[i] = silu_f(conv_at(p.q, 0, kh * s.dim + i, p.wq, 0, cv, kh * s.dim + i));
        else if (i < 2 * s.dim) sk[i - s.dim] = silu_f(conv_at(p.k, 0, kh * s.dim + i - s.dim, p.wk, 0, cv, s.qk + kh * s.dim + i - s.dim));
        else sv[i - 2 * s.dim] = silu_f(conv_at(p.v, 0, h * s.vdim + i - 2 * s.dim, p.wv, 0, cv, 2 * s.qk + h * s.vdim + i - 2 * s.dim));
    }
    __syncthreads();
    // this token's row of the ring (nobody reads it in this step); the heads of a group store the same q and k values
    for (uint32_t i = tid; i < 2 * s.dim + s.vdim; i += STEP_THREADS) {
        const uint32_t ch = i < s.dim ? kh * s.dim + i : (i < 2 * s.dim ? s.qk + kh * s.dim + i - s.dim : 2 * s.qk + h * s.vdim + i - 2 * s.dim);
        const float x = i < s.dim ? p.q[kh * s.dim + i] : (i < 2 * s.dim ? p.k[kh * s.dim + i - s.dim] : p.v[h * s.vdim + i - 2 * s.dim]);
        p.ring[(size_t)(pos % s.taps) * cv.channels + ch] = x;
    }
    const float decay = expf(p.a_log[h]);
    for (uint32_t i = warp; i < s.dim + s.vdim; i += 16) {
        if (i < s.dim) {
            const float z = row_dot(p.wa2 + (size_t)(h * s.dim + i) * p.lda2, a1, ra8, lane) + p.dt_bias[h * s.dim + i];
            if (lane == 0) sg[i] = expf(-decay * softplus_f(z));
        } else {
            const float z = row_dot(p.wg2 + (size_t)(h * s.vdim + i - s.dim) * p.ldg2, g1, rg8, lane);
            if (lane == 0) gate[i - s.dim] = sigmoid_f(z);
        }
    }
    if (warp < 3) {  // |q|^2, |k|^2, k . q before the scaling
        float v = 0.0f;
        for (uint32_t i = lane; i < s.dim; i += 32) v = fmaf(warp == 1 ? sk[i] : sq[i], warp == 0 ? sq[i] : sk[i], v);
        v = warp_sum(v);
        if (lane == 0) red[warp] = v;
    }
    __syncthreads();
    const float nq = 1.0f / (sqrtf(red[0] + UNIT_EPS) * sqrtf((float)s.dim)), nk = 1.0f / sqrtf(red[1] + UNIT_EPS), kq = red[2] * nq * nk;
    const float beta = sigmoid_f(p.b[h]);
    // partial sums of this warp's rows
    for (uint32_t c = 0; c * 32 < s.vdim; ++c) {
        const uint32_t col = lane + 32 * c;
        float ak = 0.0f, aq = 0.0f;
        if (KEEP) {
#pragma unroll
            for (int cc = 0; cc < STEP_C; ++cc)
                if (cc == (int)c)
#pragma unroll
                    for (int r = 0; r < STEP_R; ++r) {
                        const uint32_t row = warp + 16 * r;
                        if (row < s.dim) {
                            const float v = fresh ? 0.0f : keep[r][cc] * sg[row];
                            keep[r][cc] = v;
                            ak = fmaf(sk[row] * nk, v, ak);
                            aq = fmaf(sq[row] * nq, v, aq);
                        }
                    }
        } else if (col < s.vdim) {
            for (uint32_t row = warp; row < s.dim; row += 16) {
                const float v = fresh ? 0.0f : S[(size_t)row * s.vdim + col] * sg[row];
                ak = fmaf(sk[row] * nk, v, ak);
                aq = fmaf(sq[row] * nq, v, aq);
            }
        }
        if (col < s.vdim) {
            rk[warp * s.vdim + col] = ak;
            rq[warp * s.vdim + col] = aq;
        }
    }
    __syncthreads();
    for (uint32_t col = tid; col < s.vdim; col += STEP_THREADS) {
        float ak = 0.0f, aq = 0.0f;
        for (int w = 0; w < 16; ++w) {
            ak += rk[w * s.vdim + col];
            aq += rq[w * s.vdim + col];
        }
        const float u = beta * (sv[col] - ak);
        o[col] = fmaf(u, kq, aq);
        rk[col] = u;  // (only this thread reads or writes column col of the first row from here to the barrier)
    }
    __syncthreads();
    if (KEEP) {
#pragma unroll
        for (int r = 0; r < STEP_R; ++r)
#pragma unroll
            for (int c = 0; c < STEP_C; ++c) {
                const uint32_t row = warp + 16 * r, col = lane + 32 * c;
                if (row < s.dim && col < s.vdim) S[(size_t)row * s.vdim + col] = fmaf(sk[row] * nk, rk[col], keep[r][c]);
            }
    } else {
        for (uint32_t row = warp; row < s.dim; row += 16)
            for (uint32_t col = lane; col < s.vdim; col += 32) {
                const float v = fresh ? 0.0f : S[(size_t)row * s.vdim + col] * sg[row];
                S[(size_t)row * s.vdim + col] = fmaf(sk[row] * nk, rk[col], v);
            }
    }
    if (warp == 0) {
        float ss = 0.0f;
        for (uint32_t i = lane; i < s.vdim; i += 32) ss = fmaf(o[i], o[i], ss);
        const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)s.vdim + p.eps);
        for (uint32_t i = lane; i < s.vdim; i += 32) p.out[h * s.vdim + i] = o[i] * inv * p.norm[i] * gate[i];
    }
}

size_t step_smem(const DeltaShape &s, uint32_t ra, uint32_t rg) {
    return (3ull * s.dim + 35ull * s.vdim + 8 + 4 + (ra + 7) / 8 * 8 + (rg + 7) / 8 * 8) * 4;
}

}  // namespace

namespace brasa_stack {
namespace {

class ChannelDelta : public Mixer {
  public:
    bool configure(const brasa::Json &c, uint32_t width, float eps, std::string &err) override {
        if (!read_u32(c, "heads", &s_.heads, err) || !read_u32(c, "kv_heads", &s_.kv_heads, err) || !read_u32(c, "dim", &s_.dim, err) ||
            !read_u32(c, "vdim", &s_.vdim, err) || !read_u32(c, "conv", &s_.taps, err))
            return false;
        if (s_.heads % s_.kv_heads != 0) return err = "channel_delta: heads must be a multiple of kv_heads", false;
        if (s_.dim > 256 || s_.vdim > 1024) return err = "channel_delta: dim up to 256 and vdim up to 1024", false;
        s_.qk = s_.kv_heads * s_.dim;
        s_.vd = s_.heads * s_.vdim;
        width_ = width;
        eps_ = eps;
        out_width = s_.vd;
        return true;
    }

    int32_t build(Builder &b, const std::string &x) override {
        BRASA_TRY(b.matrix(x + "q", s_.qk, width_, &q_));
        BRASA_TRY(b.matrix(x + "k", s_.qk, width_, &k_));
        BRASA_TRY(b.matrix(x + "v", s_.vd, width_, &v_));
        BRASA_TRY(b.matrix(x + "b", s_.heads, width_, &b_));
        BRASA_TRY(b.matrix(x + "a1", 0, width_, &a1_));
        BRASA_TRY(b.matrix(x + "a2", s_.heads * s_.dim, a1_.rows, &a2_));
        BRASA_TRY(b.matrix(x + "g1", 0, width_, &g1_));
        BRASA_TRY(b.matrix(x + "g2", s_.vd, g1_.rows, &g2_));
        BRASA_TRY(b.matrix(x + "o", width_, s_.vd, &wo));
        BRASA_TRY(b.vector(x + "q.conv", (uint64_t)s_.qk * s_.taps, &wq_));
        BRASA_TRY(b.vector(x + "k.conv", (uint64_t)s_.qk * s_.taps, &wk_));
        BRASA_TRY(b.vector(x + "v.conv", (uint64_t)s_.vd * s_.taps, &wv_));
        BRASA_TRY(b.vector(x + "A_log", s_.heads, &a_log_));
        BRASA_TRY(b.vector(x + "dt_bias", (uint64_t)s_.heads * s_.dim, &dt_bias_));
        BRASA_TRY(b.vector(x + "norm", s_.vdim, &norm_));
        BRASA_TRY(b.get(Builder::STATE, 4ull * s_.taps * (2 * s_.qk + s_.vd), (void **)&ring_));
        BRASA_TRY(b.get(Builder::STATE, 4ull * s_.heads * s_.dim * s_.vdim, (void **)&state_));
        lay_out(b.limits.max_tokens, b.f32);
        return BRASA_OK;
    }

    uint64_t scratch_bytes(const Builder &) const override { return at_.total; }

    void project(const Run &r, std::vector<GemvProblem> &out) override {
        auto add = [&](const Weight &w, uint64_t at, uint32_t ld, bool low) {
            GemvProblem g;
            g.p.seg[0] = segment(w, r.h, r.ldh);
            g.p.rows = w.rows;
            g.p.tokens = r.tokens;
            g.p.y = r.scratch + at;
            g.p.ldy = ld;
            g.p.y_bf16 = low && !r.f32 && !r.dev_pos;
            out.push_back(g);
        };
        add(q_, at_.q, ldqk_, false);
        add(k_, at_.k, ldqk_, false);
        add(v_, at_.v, ldv_, false);
        add(b_, at_.b, ldb_, false);
        add(a1_, at_.a1, lda_, true);  // inputs of a product: bf16 where products take bf16
        add(g1_, at_.g1, ldg_, true);
    }

    int32_t mix(const Run &r) override {
        brasa_ctx *ctx = r.cmd->ctx;
        auto f = [&](uint64_t at) { return (float *)(r.scratch + at); };
        if (r.dev_pos) {
            DeltaStep p{s_, f(at_.q), f(at_.k), f(at_.v), f(at_.b), f(at_.a1), f(at_.g1), wq_, wk_, wv_, a_log_, dt_bias_, norm_, a2_.p, g2_.p,
                        a2_.cols, g2_.cols, a2_.ld, g2_.ld, ring_, state_, (float *)r.out, r.dev_pos, eps_};
            const size_t smem = step_smem(s_, a2_.cols, g2_.cols);
            const bool keep = s_.dim <= 16 * STEP_R && s_.vdim <= 32 * STEP_C;
            const void *fn = keep ? (const void *)delta_step_kernel<true> : (const void *)delta_step_kernel<false>;
            BRASA_TRY(brasa_smem_optin(ctx, fn, smem));
            if (keep) BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_step_kernel<true>, dim3(s_.heads), dim3(STEP_THREADS), smem, p));
            else BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_step_kernel<false>, dim3(s_.heads), dim3(STEP_THREADS), smem, p));
            return brasa_post_launch(r.cmd, "delta_step");
        }
        // the second factors of the decay's and the gate's projections
        LinearProblem lp[2];
        lp[0].seg[0] = segment(a2_, r.scratch + at_.a1, lda_);
        lp[0].rows = a2_.rows;
        lp[0].tokens = r.tokens;
        lp[0].y = r.scratch + at_.z;
        lp[0].ldy = ldz_;
        lp[0].bias = dt_bias_;
        lp[1].seg[0] = segment(g2_, r.scratch + at_.g1, ldg_);
        lp[1].rows = g2_.rows;
        lp[1].tokens = r.tokens;
        lp[1].y = r.scratch + at_.gate;
        lp[1].ldy = ldv_;
        BRASA_TRY(brasa_linear_launch(r.cmd, lp, 2, r.f32));
        const uint32_t channels = 2 * s_.qk + s_.vd;
        DeltaPrep pp{s_, ConvView{ring_, channels, s_.taps, r.pos0}, f(at_.q), f(at_.k), f(at_.v), f(at_.b), f(at_.z), ldqk_, ldv_, ldb_, ldz_, wq_, wk_, wv_, a_log_,
                     f(at_.qn), f(at_.kn), f(at_.vn), f(at_.g), f(at_.beta), f(at_.kq)};
        const uint32_t items = s_.kv_heads + 2 * s_.heads, gy = r.tokens < 512 ? (items + 7) / 8 : 1;
        BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_prep_kernel, dim3(r.tokens, gy), dim3(256), 0, pp));
        BRASA_TRY(brasa_post_launch(r.cmd, "delta_prep"));
        BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_ring_kernel, dim3((channels + 255) / 256), dim3(256), 0, s_, f(at_.q), f(at_.k), f(at_.v), ldqk_, ldv_, ring_,
                                               r.tokens, r.pos0));
        BRASA_TRY(brasa_post_launch(r.cmd, "delta_ring"));
        DeltaScan sp{s_, f(at_.qn), f(at_.kn), f(at_.vn), f(at_.g), f(at_.beta), f(at_.kq), state_, f(at_.o), r.tokens, r.pos0 == 0 ? 1 : 0};
        BRASA_TRY(scan(r.cmd, sp));
        const uint32_t blocks = (r.tokens * s_.heads + 7) / 8;
        if (r.f32) BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_out_kernel<float>, dim3(blocks), dim3(256), 0, f(at_.o), f(at_.gate), ldv_, norm_, (float *)r.out, r.ldo,
                                                          s_.heads, s_.vdim, r.tokens, eps_));
        else BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_out_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, f(at_.o), f(at_.gate), ldv_, norm_,
                                                    (__nv_bfloat16 *)r.out, r.ldo, s_.heads, s_.vdim, r.tokens, eps_));
        return brasa_post_launch(r.cmd, "delta_out");
    }

  private:
    int32_t scan(brasa_cmd *cmd, const DeltaScan &p) {
        brasa_ctx *ctx = cmd->ctx;
        // two columns per thread when that still fills the SMs
        const bool two = s_.heads * ((s_.vdim + 31) / 32) >= (uint32_t)ctx->sm_count / 2;
        const dim3 grid(s_.heads, (s_.vdim + (two ? 31 : 15)) / (two ? 32 : 16));
#define SCAN(R)                                                                                                              \
    do {                                                                                                                     \
        if (two) BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_scan_kernel<R, 2>, grid, dim3(256), 0, p));               \
        else BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_scan_kernel<R, 1>, grid, dim3(256), 0, p));                   \
    } while (0)
        if (s_.dim <= 64) SCAN(4);
        else if (s_.dim <= 128) SCAN(8);
        else BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_scan_kernel<16, 1>, dim3(s_.heads, (s_.vdim + 15) / 16), dim3(256), 0, p));
#undef SCAN
        return brasa_post_launch(cmd, "delta_scan");
    }

    void lay_out(uint64_t t, bool f32) {
        ldqk_ = up8(s_.qk);
        ldv_ = up8(s_.vd);
        ldb_ = up8(s_.heads);
        lda_ = up8(a1_.rows);
        ldg_ = up8(g1_.rows);
        ldz_ = up8(s_.heads * s_.dim);
        (void)f32;
        Carver c;
        at_.q = c.take(4 * t * ldqk_);
        at_.k = c.take(4 * t * ldqk_);
        at_.v = c.take(4 * t * ldv_);
        at_.b = c.take(4 * t * ldb_);
        at_.a1 = c.take(4 * t * lda_);
        at_.g1 = c.take(4 * t * ldg_);
        at_.z = c.take(4 * t * ldz_);
        at_.gate = c.take(4 * t * ldv_);
        at_.qn = c.take(4 * t * s_.qk);
        at_.kn = c.take(4 * t * s_.qk);
        at_.vn = c.take(4 * t * s_.vd);
        at_.g = c.take(4 * t * s_.heads * s_.dim);
        at_.beta = c.take(4 * t * s_.heads);
        at_.kq = c.take(4 * t * s_.kv_heads);
        at_.o = c.take(4 * t * s_.vd);
        at_.total = c.at;
    }

    DeltaShape s_{};
    uint32_t width_ = 0, ldqk_ = 0, ldv_ = 0, ldb_ = 0, lda_ = 0, ldg_ = 0, ldz_ = 0;
    float eps_ = 0.0f;
    Weight q_, k_, v_, b_, a1_, a2_, g1_, g2_;
    const float *wq_ = nullptr, *wk_ = nullptr, *wv_ = nullptr, *a_log_ = nullptr, *dt_bias_ = nullptr, *norm_ = nullptr;
    float *ring_ = nullptr, *state_ = nullptr;
    struct {
        uint64_t q, k, v, b, a1, g1, z, gate, qn, kn, vn, g, beta, kq, o, total;
    } at_{};
};

}  // namespace

std::unique_ptr<Mixer> make_channel_delta() { return std::unique_ptr<Mixer>(new ChannelDelta()); }

}  // namespace brasa_stack
