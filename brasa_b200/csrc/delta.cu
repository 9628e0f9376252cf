// Gated delta rule with one decay per key channel ("channel_delta"), a recurrent mixer. A head keeps a matrix S [dim][vdim] of
// what each key direction stands for. A token fades the rows of S by its decays g, reads what its key k finds there, moves that
// towards its value v by the fraction beta, and its query q reads the result:
//   F = diag(g) S_old,  u = beta (v - F^T k),  S_new = F + k u^T,  o = S_new^T q
// q, k and v come out of a short causal convolution and silu, q and k as unit vectors, g out of a softplus.
//
// Many tokens: chunks of 16, everything that does not depend on the state for all chunks side by side, then the state through
// the chunks (below). One token: delta_step_kernel does all of it, one block per head. Everything is f32 FMA.
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

// ---- many tokens -------------------------------------------------------------------------------------------------------
// Tokens go in chunks of CH. Inside a chunk write c_t for the product of the decays up to token t and let
//   A[t][s] = sum k_t k_s c_t / c_s (s < t),  B[t][s] = sum q_t k_s c_t / c_s (s <= t)      (sums over key channels)
// Unrolling the recurrence over the chunk gives, with the state S before it,
//   U = T (V - K' S),  T = (I + diag(beta) A)^-1 diag(beta),  K'_t = c_t k_t
//   O = Q' S + B U,  Q'_t = c_t q_t
//   S_next = diag(c_last) S + K''^T U,  K''_s = k_s c_last / c_s
// T and B do not depend on the state: delta_chunk_kernel forms them for all chunks side by side, together with q, k, v and g.
// delta_scan_kernel then carries the state through the chunks with products instead of one reduction per token. The ratios
// c_t / c_s are always formed as products of the decays between s and t, never by division.
constexpr uint32_t CH = 16;

struct DeltaChunk {
    DeltaShape s;
    ConvView cv;
    const float *q, *k, *v, *b, *z;  // products [tokens][ld]
    uint32_t ldqk, ldv, ldb, ldz, tokens;
    const float *wq, *wk, *wv, *a_log;
    float *qn, *kn, *vn, *g, *tb;    // [tokens][qk], [qk], [vd], [heads * dim]; [chunks][heads][T, B][CH][CH]
};

// convolution and silu of one channel for the chunk's tokens, handed to put(t, value)
template <typename Put>
__device__ __forceinline__ void conv_chunk(const float *x, uint32_t ldx, uint32_t c, const float *w, uint32_t t0, uint32_t n, const ConvView &cv, uint32_t ch, Put put) {
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
        float in[CH];
#pragma unroll
        for (uint32_t t = 0; t < CH; ++t) in[t] = t < n ? x[(size_t)(t0 + t) * ldx + c] : 0.0f;
#pragma unroll
        for (uint32_t t = 0; t < CH; ++t) {
            xr[0] = xr[1];
            xr[1] = xr[2];
            xr[2] = xr[3];
            xr[3] = in[t];
            if (t < n) put(t, silu_f(fmaf(xr[3], wr[3], fmaf(xr[2], wr[2], fmaf(xr[1], wr[1], xr[0] * wr[0])))));
        }
    } else {
        for (uint32_t t = 0; t < n; ++t) put(t, silu_f(conv_at(x, ldx, c, w, t0 + t, cv, ch)));
    }
}

// Block: one chunk of one kv head and the heads that share it.
__global__ void __launch_bounds__(256) delta_chunk_kernel(DeltaChunk p) {
    extern __shared__ __align__(16) float sm[];
    const DeltaShape s = p.s;
    float *sq = sm, *sk = sq + CH * s.dim, *sg = sk + CH * s.dim;
    __shared__ float A[CH][CH + 1], B[CH][CH], T[CH][CH + 1], beta[CH];
    const uint32_t chunk = blockIdx.x, t0 = chunk * CH, n = min(CH, p.tokens - t0), kh = blockIdx.y, group = s.heads / s.kv_heads;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    pdl_wait();
    pdl_launch();
    for (uint32_t i = tid; i < 2 * s.dim; i += 256) {
        const bool isk = i >= s.dim;
        const uint32_t e = isk ? i - s.dim : i, c = kh * s.dim + e;
        float *dst = (isk ? sk : sq) + e;
        conv_chunk(isk ? p.k : p.q, p.ldqk, c, isk ? p.wk : p.wq, t0, n, p.cv, (isk ? s.qk : 0u) + c, [&](uint32_t t, float v) { dst[t * s.dim] = v; });
        for (uint32_t t = n; t < CH; ++t) dst[t * s.dim] = 0.0f;
    }
    __syncthreads();
    for (uint32_t i = warp; i < 2 * n; i += 8) {  // unit vectors; q also over the root of its size
        float *v = (i & 1 ? sk : sq) + (i >> 1) * s.dim, *out = (i & 1 ? p.kn : p.qn) + (size_t)(t0 + (i >> 1)) * s.qk + kh * s.dim;
        float ss = 0.0f;
        for (uint32_t e = lane; e < s.dim; e += 32) ss = fmaf(v[e], v[e], ss);
        ss = 1.0f / sqrtf(warp_sum(ss) + UNIT_EPS);
        if (!(i & 1)) ss /= sqrtf((float)s.dim);
        for (uint32_t e = lane; e < s.dim; e += 32) {
            v[e] *= ss;
            out[e] = v[e];
        }
    }
    for (uint32_t hh = 0; hh < group; ++hh) {
        const uint32_t h = kh * group + hh;
        const float a = expf(p.a_log[h]);
        for (uint32_t i = tid; i < s.vdim; i += 256) {
            const uint32_t c = h * s.vdim + i;
            conv_chunk(p.v, p.ldv, c, p.wv, t0, n, p.cv, 2 * s.qk + c, [&](uint32_t t, float v) { p.vn[(size_t)(t0 + t) * s.vd + c] = v; });
        }
        for (uint32_t t = warp; t < CH; t += 8)
            for (uint32_t e = lane; e < s.dim; e += 32) {
                float g = 1.0f;
                if (t < n) {
                    g = expf(-a * softplus_f(p.z[(size_t)(t0 + t) * p.ldz + h * s.dim + e]));
                    p.g[((size_t)(t0 + t) * s.heads + h) * s.dim + e] = g;
                }
                sg[t * s.dim + e] = g;
            }
        if (tid < CH) beta[tid] = tid < n ? sigmoid_f(p.b[(size_t)(t0 + tid) * p.ldb + h]) : 0.0f;
        __syncthreads();
        // A and B: warp w takes the columns s = w and 15 - w; lanes run along the channels with the product of the decays so far
        for (int half = 0; half < 2; ++half) {
            const uint32_t col = half ? CH - 1 - warp : warp;
            float ks[8], run[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const uint32_t e = lane + 32 * j;
                ks[j] = e < s.dim ? sk[col * s.dim + e] : 0.0f;
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) run[j] = ks[j];
            for (uint32_t t = 0; t < col; ++t)
                if (lane == 0) A[t][col] = B[t][col] = 0.0f;
            for (uint32_t t = col; t < CH; ++t) {
                float sa = 0.0f, sb = 0.0f;
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    const uint32_t e = lane + 32 * j;
                    if (e < s.dim) {
                        if (t > col) run[j] *= sg[t * s.dim + e];
                        sa = fmaf(sk[t * s.dim + e], run[j], sa);
                        sb = fmaf(sq[t * s.dim + e], run[j], sb);
                    }
                }
                sa = warp_sum(sa);
                sb = warp_sum(sb);
                if (lane == 0) {
                    A[t][col] = t > col ? sa : 0.0f;
                    B[t][col] = sb;
                }
            }
        }
        __syncthreads();
        if (tid < CH) {  // column tid of T by forward substitution
            for (uint32_t t = 0; t < CH; ++t) {
                float v = t == tid ? 1.0f : 0.0f;
                for (uint32_t r = tid; r < t; ++r) v = fmaf(-A[t][r], T[r][tid], v);
                T[t][tid] = t < tid ? 0.0f : beta[t] * v;
            }
        }
        __syncthreads();
        float *tb = p.tb + ((size_t)chunk * s.heads + h) * 2 * CH * CH;
        tb[tid] = T[tid >> 4][tid & 15];
        tb[CH * CH + tid] = B[tid >> 4][tid & 15];
        __syncthreads();
    }
}

struct DeltaScan {
    DeltaShape s;
    const float *qn, *kn, *vn, *g, *tb;
    const float *q, *k, *v;  // the convolution's inputs, whose last rows go to the ring
    uint32_t ldqk, ldv;
    float *ring;
    float *state;  // [heads][dim][vdim]
    float *o;      // [tokens][vd]
    uint32_t tokens, pos0;
};

__device__ __forceinline__ void cp4(float *dst, const float *src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp16(float *dst, const float *src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

// D: key channels rounded up to 64, 128 or 256; CB: state columns of a block, 16 or 32.
template <int D, int CB>
struct ScanShape {
    static constexpr uint32_t IN = 3 * CH * D + CH * CB + 2 * CH * CH;  // a stage: q, k, g, v, T, B
    static constexpr uint32_t LDA = 2 * CH + 4;                         // K' and Q' as [channel][32 rows], padded
    static constexpr uint32_t FLOATS = 2 * IN + D * LDA + CH * D + D + D * CB + 8 * 2 * CH * CB + 2 * CH * CB;
};

template <int D, int CB>
__global__ void __launch_bounds__(256, 1) delta_scan_kernel(DeltaScan p) {
    using Sh = ScanShape<D, CB>;
    constexpr uint32_t LDA = Sh::LDA, KW = D / 8, CPL = CB / 4, TILES = D / 4 * (CB / 4), TPT = (TILES + 255) / 256;
    extern __shared__ __align__(16) float sm[];
    float *in = sm, *at = in + 2 * Sh::IN, *kend = at + D * LDA, *cend = kend + CH * D, *S = cend + D, *red = S + D * CB, *X = red + 8 * 2 * CH * CB, *U = X + CH * CB;
    const DeltaShape s = p.s;
    const uint32_t h = blockIdx.x, kh = h / (s.heads / s.kv_heads), c0 = blockIdx.y * CB;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    for (uint32_t i = tid; i < 2 * Sh::IN; i += 256) in[i] = 0.0f;  // padding: zero k and q leave padded rows of the state at zero
    __syncthreads();
    pdl_wait();
    pdl_launch();
    {  // the run's last inputs of the convolution into the ring (the kernel that read the older ones has finished)
        const uint32_t channels = 2 * s.qk + s.vd, n = min(p.tokens, s.taps), blocks = gridDim.x * gridDim.y;
        for (uint32_t ch = (blockIdx.y * gridDim.x + blockIdx.x) * 256 + tid; ch < channels; ch += blocks * 256)
            for (uint32_t t = p.tokens - n; t < p.tokens; ++t) {
                const float x = ch < s.qk ? p.q[(size_t)t * p.ldqk + ch] : (ch < 2 * s.qk ? p.k[(size_t)t * p.ldqk + ch - s.qk] : p.v[(size_t)t * p.ldv + ch - 2 * s.qk]);
                p.ring[(size_t)((p.pos0 + t) % s.taps) * channels + ch] = x;
            }
    }
    const uint32_t ncol = min((uint32_t)CB, s.vdim - c0);
    // this thread's 4 x 4 tiles of the state, kept in registers; S in shared memory is what the products read
    float st[TPT][4][4];
#pragma unroll
    for (uint32_t u = 0; u < TPT; ++u) {
        const uint32_t tile = tid + 256 * u, r0 = tile / (CB / 4) * 4, k0 = tile % (CB / 4) * 4;
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const uint32_t row = r0 + i, col = c0 + k0 + j;
                st[u][i][j] = (tile < TILES && p.pos0 != 0 && row < s.dim && col < s.vdim) ? p.state[((size_t)h * s.dim + row) * s.vdim + col] : 0.0f;
                if (tile < TILES) S[(r0 + i) * CB + k0 + j] = st[u][i][j];
            }
    }
    const bool vec = (s.dim & 3) == 0, vecv = (s.vdim & 3) == 0;
    auto fetch = [&](uint32_t chunk) {
        float *b = in + (chunk & 1) * Sh::IN;
        const uint32_t t0 = chunk * CH, n = min(CH, p.tokens - t0);
        if (vec) {
            for (uint32_t t = warp; t < n; t += 8)
                for (uint32_t e = lane * 4; e < s.dim; e += 128) {
                    cp16(b + t * D + e, p.qn + (size_t)(t0 + t) * s.qk + kh * s.dim + e);
                    cp16(b + (CH + t) * D + e, p.kn + (size_t)(t0 + t) * s.qk + kh * s.dim + e);
                    cp16(b + (2 * CH + t) * D + e, p.g + ((size_t)(t0 + t) * s.heads + h) * s.dim + e);
                }
        } else {
            for (uint32_t t = warp; t < n; t += 8)
                for (uint32_t e = lane; e < s.dim; e += 32) {
                    cp4(b + t * D + e, p.qn + (size_t)(t0 + t) * s.qk + kh * s.dim + e);
                    cp4(b + (CH + t) * D + e, p.kn + (size_t)(t0 + t) * s.qk + kh * s.dim + e);
                    cp4(b + (2 * CH + t) * D + e, p.g + ((size_t)(t0 + t) * s.heads + h) * s.dim + e);
                }
        }
        float *bv = b + 3 * CH * D;
        for (uint32_t t = warp; t < n; t += 8)
            for (uint32_t e = lane; e < ncol; e += 32) cp4(bv + t * CB + e, p.vn + (size_t)(t0 + t) * s.vd + h * s.vdim + c0 + e);
        if (tid < 2 * CH * CH / 4) cp16(bv + CH * CB + 4 * tid, p.tb + ((size_t)chunk * s.heads + h) * 2 * CH * CH + 4 * tid);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const uint32_t chunks = (p.tokens + CH - 1) / CH;
    fetch(0);
    for (uint32_t chunk = 0; chunk < chunks; ++chunk) {
        float *b = in + (chunk & 1) * Sh::IN, *bv = b + 3 * CH * D;
        const float *bt = bv + CH * CB, *bb = bt + CH * CH;
        const uint32_t t0 = chunk * CH, n = min(CH, p.tokens - t0);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // the chunk's inputs have arrived; everything of the chunk before has been read
        if (chunk + 1 < chunks) fetch(chunk + 1);
        // K', Q', K'' and the chunk's whole decay, one channel per thread (tokens past the end: k = q = 0, no decay)
        for (uint32_t c = tid; c < 2 * D; c += 256) {
            const uint32_t e = c < D ? c : c - D;
            if (c < D) {
                float run = 1.0f;
#pragma unroll
                for (uint32_t t4 = 0; t4 < CH; t4 += 4) {
                    float kk[4], qq[4];
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const uint32_t t = t4 + i;
                        if (t < n) run *= b[(2 * CH + t) * D + e];
                        qq[i] = t < n ? b[t * D + e] * run : 0.0f;
                        kk[i] = t < n ? b[(CH + t) * D + e] * run : 0.0f;
                    }
                    *reinterpret_cast<float4 *>(at + e * LDA + t4) = make_float4(kk[0], kk[1], kk[2], kk[3]);
                    *reinterpret_cast<float4 *>(at + e * LDA + CH + t4) = make_float4(qq[0], qq[1], qq[2], qq[3]);
                }
            } else {
                float run = 1.0f;
#pragma unroll
                for (int t = CH - 1; t >= 0; --t) {
                    const bool live = (uint32_t)t < n;
                    kend[t * D + e] = live ? b[(CH + t) * D + e] * run : 0.0f;
                    if (live) run *= b[(2 * CH + t) * D + e];
                }
                cend[e] = run;
            }
        }
        __syncthreads();
        {  // [K'; Q'] S: warp w sums over its share of the channels; lane = 4 of the 32 rows x CPL columns
            float acc[4][CPL] = {};
            const uint32_t r4 = (lane >> 2) * 4, cl = (lane & 3) * CPL;
#pragma unroll 4
            for (uint32_t k = warp * KW; k < (warp + 1) * KW; ++k) {
                const float4 a = *reinterpret_cast<const float4 *>(at + k * LDA + r4);
                const float av[4] = {a.x, a.y, a.z, a.w};
                float sv[CPL];
#pragma unroll
                for (uint32_t j = 0; j < CPL; j += 4) {
                    const float4 v = *reinterpret_cast<const float4 *>(S + k * CB + cl + j);
                    sv[j] = v.x;
                    sv[j + 1] = v.y;
                    sv[j + 2] = v.z;
                    sv[j + 3] = v.w;
                }
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (uint32_t j = 0; j < CPL; ++j) acc[i][j] = fmaf(av[i], sv[j], acc[i][j]);
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (uint32_t j = 0; j < CPL; j += 4)
                    *reinterpret_cast<float4 *>(red + (warp * 2 * CH + r4 + i) * CB + cl + j) = make_float4(acc[i][j], acc[i][j + 1], acc[i][j + 2], acc[i][j + 3]);
        }
        __syncthreads();
        // the sums over the warps: rows 0-15 become X = V - K' S, rows 16-31 stay with their thread (Q' S)
        const uint32_t row = tid / (CB / 4), k4 = tid % (CB / 4) * 4;
        const bool mine = row < 2 * CH;
        float o[4] = {};
        if (mine) {
#pragma unroll
            for (int w = 0; w < 8; ++w) {
                const float4 v = *reinterpret_cast<const float4 *>(red + (w * 2 * CH + row) * CB + k4);
                o[0] += v.x;
                o[1] += v.y;
                o[2] += v.z;
                o[3] += v.w;
            }
            if (row < CH) {
                const float4 v = *reinterpret_cast<const float4 *>(bv + row * CB + k4);
                *reinterpret_cast<float4 *>(X + row * CB + k4) = row < n ? make_float4(v.x - o[0], v.y - o[1], v.z - o[2], v.w - o[3]) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
        }
        __syncthreads();
        if (mine && row < CH) {
            float u[4] = {};
#pragma unroll
            for (uint32_t r = 0; r < CH; ++r) {
                const float t = bt[row * CH + r];
                const float4 x = *reinterpret_cast<const float4 *>(X + r * CB + k4);
                u[0] = fmaf(t, x.x, u[0]);
                u[1] = fmaf(t, x.y, u[1]);
                u[2] = fmaf(t, x.z, u[2]);
                u[3] = fmaf(t, x.w, u[3]);
            }
            *reinterpret_cast<float4 *>(U + row * CB + k4) = make_float4(u[0], u[1], u[2], u[3]);
        }
        __syncthreads();
        if (mine && row >= CH && row - CH < n) {
            const uint32_t t = row - CH;
#pragma unroll
            for (uint32_t r = 0; r < CH; ++r) {
                const float w = bb[t * CH + r];
                const float4 u = *reinterpret_cast<const float4 *>(U + r * CB + k4);
                o[0] = fmaf(w, u.x, o[0]);
                o[1] = fmaf(w, u.y, o[1]);
                o[2] = fmaf(w, u.z, o[2]);
                o[3] = fmaf(w, u.w, o[3]);
            }
            float *dst = p.o + (size_t)(t0 + t) * s.vd + h * s.vdim + c0 + k4;
            if (vecv && k4 + 4 <= ncol) *reinterpret_cast<float4 *>(dst) = make_float4(o[0], o[1], o[2], o[3]);
            else
                for (uint32_t j = 0; j < 4; ++j)
                    if (k4 + j < ncol) dst[j] = o[j];
        }
#pragma unroll
        for (uint32_t u = 0; u < TPT; ++u) {
            const uint32_t tile = tid + 256 * u, r0 = tile / (CB / 4) * 4, kc = tile % (CB / 4) * 4;
            if (tile < TILES) {
                const float4 ce = *reinterpret_cast<const float4 *>(cend + r0);
                const float cv[4] = {ce.x, ce.y, ce.z, ce.w};
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int j = 0; j < 4; ++j) st[u][i][j] *= cv[i];
#pragma unroll
                for (uint32_t r = 0; r < CH; ++r) {
                    const float4 kv = *reinterpret_cast<const float4 *>(kend + r * D + r0), uv = *reinterpret_cast<const float4 *>(U + r * CB + kc);
                    const float ka[4] = {kv.x, kv.y, kv.z, kv.w}, ua[4] = {uv.x, uv.y, uv.z, uv.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i)
#pragma unroll
                        for (int j = 0; j < 4; ++j) st[u][i][j] = fmaf(ka[i], ua[j], st[u][i][j]);
                }
#pragma unroll
                for (int i = 0; i < 4; ++i) *reinterpret_cast<float4 *>(S + (r0 + i) * CB + kc) = make_float4(st[u][i][0], st[u][i][1], st[u][i][2], st[u][i][3]);
            }
        }
    }
#pragma unroll
    for (uint32_t u = 0; u < TPT; ++u) {
        const uint32_t tile = tid + 256 * u, r0 = tile / (CB / 4) * 4, kc = tile % (CB / 4) * 4;
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const uint32_t row = r0 + i, col = c0 + kc + j;
                if (tile < TILES && row < s.dim && col < s.vdim) p.state[((size_t)h * s.dim + row) * s.vdim + col] = st[u][i][j];
            }
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
        DeltaChunk cp{s_, ConvView{ring_, channels, s_.taps, r.pos0}, f(at_.q), f(at_.k), f(at_.v), f(at_.b), f(at_.z), ldqk_, ldv_, ldb_, ldz_, r.tokens, wq_, wk_, wv_, a_log_,
                      f(at_.qn), f(at_.kn), f(at_.vn), f(at_.g), f(at_.tb)};
        const size_t csm = 3ull * CH * s_.dim * 4;
        BRASA_TRY(brasa_smem_optin(ctx, (const void *)delta_chunk_kernel, csm));
        BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_chunk_kernel, dim3((r.tokens + CH - 1) / CH, s_.kv_heads), dim3(256), csm, cp));
        BRASA_TRY(brasa_post_launch(r.cmd, "delta_chunk"));
        DeltaScan sp{s_, f(at_.qn), f(at_.kn), f(at_.vn), f(at_.g), f(at_.tb), f(at_.q), f(at_.k), f(at_.v), ldqk_, ldv_, ring_, state_, f(at_.o), r.tokens, r.pos0};
        BRASA_TRY(scan(r.cmd, sp));
        const uint32_t blocks = (r.tokens * s_.heads + 7) / 8;
        if (r.f32) BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_out_kernel<float>, dim3(blocks), dim3(256), 0, f(at_.o), f(at_.gate), ldv_, norm_, (float *)r.out, r.ldo,
                                                          s_.heads, s_.vdim, r.tokens, eps_));
        else BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_out_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, f(at_.o), f(at_.gate), ldv_, norm_,
                                                    (__nv_bfloat16 *)r.out, r.ldo, s_.heads, s_.vdim, r.tokens, eps_));
        return brasa_post_launch(r.cmd, "delta_out");
    }

  private:
    template <int D, int CB>
    int32_t scan_as(brasa_cmd *cmd, const DeltaScan &p) {
        brasa_ctx *ctx = cmd->ctx;
        const size_t smem = (size_t)ScanShape<D, CB>::FLOATS * 4;
        BRASA_TRY(brasa_smem_optin(ctx, (const void *)delta_scan_kernel<D, CB>, smem));
        BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_scan_kernel<D, CB>, dim3(s_.heads, (s_.vdim + CB - 1) / CB), dim3(256), smem, p));
        return brasa_post_launch(cmd, "delta_scan");
    }
    int32_t scan(brasa_cmd *cmd, const DeltaScan &p) {
        // wide blocks when they still cover most of the SMs
        const bool wide = s_.heads * ((s_.vdim + 31) / 32) * 5 >= (uint32_t)cmd->ctx->sm_count * 4;
        if (s_.dim <= 64) return wide ? scan_as<64, 32>(cmd, p) : scan_as<64, 16>(cmd, p);
        if (s_.dim <= 128) return wide ? scan_as<128, 32>(cmd, p) : scan_as<128, 16>(cmd, p);
        return scan_as<256, 16>(cmd, p);
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
        at_.tb = c.take(4ull * ((t + CH - 1) / CH) * s_.heads * 2 * CH * CH);
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
        uint64_t q, k, v, b, a1, g1, z, gate, qn, kn, vn, g, tb, o, total;
    } at_{};
};

}  // namespace

std::unique_ptr<Mixer> make_channel_delta() { return std::unique_ptr<Mixer>(new ChannelDelta()); }

}  // namespace brasa_stack
