// Gated delta rule, a recurrent mixer. A head keeps a matrix S [dim][vdim] of what each key direction stands for. A token fades
// the rows of S by its decays g, reads what its key k finds there, moves that towards its value v by the fraction beta, and its
// query q reads the result:
//   F = diag(g) S_old,  u = beta (v - F^T k),  S_new = F + k u^T,  o = S_new^T q
// q, k and v come out of a short causal convolution and silu, q and k as unit vectors, g out of a softplus.
// Two forms: "channel_delta" has one decay per key channel and a sigmoid output gate, both out of low-rank projections; "delta"
// has one decay per head (HD below) and a silu output gate, both out of plain projections.
//
// Many tokens: chunks of 16, everything that does not depend on the state for all chunks side by side, then the state through
// the chunks (below). One token: delta_step_kernel does all of it, one block per head. Everything is f32 FMA.
//
// Per-sequence state: S [heads][dim][vdim] and the convolution's inputs as a ring of `taps` rows, position p in row p % taps
// (one more row than needed, so that a step can store its own row while others still read the older ones). A sequence
// starts at position 0 by ignoring both.
#include <cuda_bf16.h>

#include "conv_device.cuh"
#include "stack.h"
#include "tc_device.cuh"

using namespace brasa_dev;

namespace {

constexpr float UNIT_EPS = 1e-6f;

struct DeltaShape {
    uint32_t heads, kv_heads, dim, vdim, taps;
    uint32_t qk;  // kv_heads * dim
    uint32_t vd;  // heads * vdim
};

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
    float *qn, *kn, *vn, *g, *tb;    // [tokens][qk], [qk], [vd], [heads * dim] (HD: [heads]); [chunks][heads][T, B][CH][CH]
};

// E consecutive floats of shared memory
template <int E>
__device__ __forceinline__ void load_run(const float *p, float v[E]) {
    if (E == 2) {
        const float2 a = *reinterpret_cast<const float2 *>(p);
        v[0] = a.x;
        v[1] = a.y;
    } else {
#pragma unroll
        for (int j = 0; j < E; j += 4) {
            const float4 a = *reinterpret_cast<const float4 *>(p + j);
            v[j] = a.x;
            v[j + 1] = a.y;
            v[j + 2] = a.z;
            v[j + 3] = a.w;
        }
    }
}

// Block: one chunk of one head. E consecutive key channels per lane: dim up to 32 E.
template <int E, bool HD>
__global__ void __launch_bounds__(256) delta_chunk_kernel(DeltaChunk p) {
    constexpr uint32_t D = 32 * E;
    extern __shared__ __align__(16) float sm[];
    const DeltaShape s = p.s;
    float *sq = sm, *sk = sq + CH * D, *sg = sk + CH * D;
    __shared__ float B[CH][CH], beta[CH], gh[CH];
    __shared__ __align__(16) float A[CH][CH];
    const uint32_t chunk = blockIdx.x, t0 = chunk * CH, n = min(CH, p.tokens - t0), h = blockIdx.y, group = s.heads / s.kv_heads, kh = h / group;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    pdl_wait();
    pdl_launch();
    for (uint32_t i = tid; i < 2 * D; i += 256) {
        const bool isk = i >= D;
        const uint32_t e = isk ? i - D : i, c = kh * s.dim + e;
        float *dst = (isk ? sk : sq) + e;
        uint32_t t = 0;
        if (e < s.dim) {
            conv_chunk(isk ? p.k : p.q, p.ldqk, c, isk ? p.wk : p.wq, 0.0f, t0, n, p.cv, (isk ? s.qk : 0u) + c, [&](uint32_t tt, float v) { dst[tt * D] = v; });
            t = n;
        }
        for (; t < CH; ++t) dst[t * D] = 0.0f;
    }
    {
        const float a = expf(p.a_log[h]);
        if (HD) {
            if (tid < CH) {
                gh[tid] = tid < n ? expf(-a * softplus_f(p.z[(size_t)(t0 + tid) * p.ldz + h])) : 1.0f;
                if (tid < n) p.g[(size_t)(t0 + tid) * s.heads + h] = gh[tid];
            }
        } else {
            for (uint32_t t = warp; t < CH; t += 8)
#pragma unroll
                for (int j = 0; j < E; ++j) {
                    const uint32_t e = lane + 32 * j;
                    float g = 1.0f;
                    if (t < n && e < s.dim) {
                        g = expf(-a * softplus_f(p.z[(size_t)(t0 + t) * p.ldz + h * s.dim + e]));
                        p.g[((size_t)(t0 + t) * s.heads + h) * s.dim + e] = g;
                    }
                    sg[t * D + e] = g;
                }
        }
        if (tid < CH) beta[tid] = tid < n ? sigmoid_f(p.b[(size_t)(t0 + tid) * p.ldb + h]) : 0.0f;
    }
    __syncthreads();
    for (uint32_t i = warp; i < 2 * n; i += 8) {  // unit vectors; q also over the root of its size
        float *v = (i & 1 ? sk : sq) + (i >> 1) * D, *out = (i & 1 ? p.kn : p.qn) + (size_t)(t0 + (i >> 1)) * s.qk + kh * s.dim;
        float x[E], ss = 0.0f;
#pragma unroll
        for (int j = 0; j < E; ++j) {
            x[j] = v[lane + 32 * j];
            ss = fmaf(x[j], x[j], ss);
        }
        ss = 1.0f / sqrtf(warp_sum(ss) + UNIT_EPS);
        if (!(i & 1)) ss /= sqrtf((float)s.dim);
#pragma unroll
        for (int j = 0; j < E; ++j) {
            v[lane + 32 * j] = x[j] * ss;
            if (h % group == 0 && lane + 32 * j < s.dim) out[lane + 32 * j] = x[j] * ss;
        }
    }
    __syncthreads();
    // A and B: warp w takes the columns s = w and 15 - w; a lane holds E channels of k_s times the decays so far, sums of all t
    // are kept apart and reduced over the lanes together at the end
#pragma unroll 1
    for (int half = 0; half < 2; ++half) {
        const uint32_t col = half ? CH - 1 - warp : warp;
        float run[E], acc[2 * CH];
        load_run<E>(sk + col * D + lane * E, run);
#pragma unroll
        for (uint32_t t = 0; t < CH; ++t) {
            acc[2 * t] = acc[2 * t + 1] = 0.0f;
            if (t >= col) {
                float kk[E], qq[E];
                load_run<E>(sk + t * D + lane * E, kk);
                load_run<E>(sq + t * D + lane * E, qq);
                if (HD) {
                    if (t > col)
#pragma unroll
                        for (int j = 0; j < E; ++j) run[j] *= gh[t];
                } else if (t > col) {
                    float gg[E];
                    load_run<E>(sg + t * D + lane * E, gg);
#pragma unroll
                    for (int j = 0; j < E; ++j) run[j] *= gg[j];
                }
#pragma unroll
                for (int j = 0; j < E; ++j) {
                    acc[2 * t] = fmaf(kk[j], run[j], acc[2 * t]);
                    acc[2 * t + 1] = fmaf(qq[j], run[j], acc[2 * t + 1]);
                }
            }
        }
        // 32 values over 32 lanes: lane i ends up with value i
#pragma unroll
        for (int w = CH; w >= 1; w >>= 1) {
            const bool up = lane & w;
#pragma unroll
            for (int i = 0; i < w; ++i) {
                const float give = up ? acc[i] : acc[i + w], keep = up ? acc[i + w] : acc[i];
                acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, w);
            }
        }
        const uint32_t t = lane >> 1;
        if (lane & 1) B[t][col] = acc[0];
        else A[t][col] = t > col ? acc[0] : 0.0f;
    }
    __syncthreads();
    float *tb = p.tb + ((size_t)chunk * s.heads + h) * 2 * CH * CH;
    if (warp == 0) {
        if (lane < CH) {  // column `lane` of T by forward substitution
            float T[CH];
#pragma unroll
            for (uint32_t t = 0; t < CH; ++t) {
                float v = t == lane ? 1.0f : 0.0f;
#pragma unroll
                for (uint32_t r = 0; r < t; ++r) v = fmaf(-A[t][r], T[r], v);
                T[t] = beta[t] * v;
                tb[t * CH + lane] = T[t];
            }
        }
    } else {
        for (uint32_t i = tid - 32; i < CH * CH; i += 224) tb[CH * CH + i] = B[i >> 4][i & 15];
        for (uint32_t i = tid - 32; i < s.vdim; i += 224) {
            const uint32_t c = h * s.vdim + i;
            conv_chunk(p.v, p.ldv, c, p.wv, 0.0f, t0, n, p.cv, 2 * s.qk + c, [&](uint32_t t, float v) { p.vn[(size_t)(t0 + t) * s.vd + c] = v; });
        }
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

// The run's last inputs of the convolution into the ring (the kernel that read the older ones has finished).
__device__ __forceinline__ void store_ring(const DeltaScan &p, uint32_t threads) {
    const DeltaShape &s = p.s;
    const uint32_t channels = 2 * s.qk + s.vd, n = min(p.tokens, s.taps), step = gridDim.x * gridDim.y * threads;
    for (uint32_t ch = (blockIdx.y * gridDim.x + blockIdx.x) * threads + threadIdx.x; ch < channels; ch += step)
        for (uint32_t t = p.tokens - n; t < p.tokens; ++t) {
            const float x = ch < s.qk ? p.q[(size_t)t * p.ldqk + ch] : (ch < 2 * s.qk ? p.k[(size_t)t * p.ldqk + ch - s.qk] : p.v[(size_t)t * p.ldv + ch - 2 * s.qk]);
            p.ring[(size_t)((p.pos0 + t) % s.taps) * channels + ch] = x;
        }
}

// The state through the chunks in f32 FMA (the 32-bit mode, and key sizes above 128). D: key channels rounded up to 64, 128 or
// 256; CB: state columns of a block, 16 or 32.
template <int D, int CB>
struct ScanShape {
    static constexpr uint32_t IN = 3 * CH * D + CH * CB + 2 * CH * CH;  // a stage: q, k, g, v, T, B
    static constexpr uint32_t LDA = 2 * CH + 4;                         // K' and Q' as [channel][32 rows], padded
    static constexpr uint32_t FLOATS = 2 * IN + D * LDA + CH * D + D + D * CB + 8 * 2 * CH * CB + 2 * CH * CB;
};

template <int D, int CB, bool HD>
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
    store_ring(p, 256);
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
                    if (!HD) cp16(b + (2 * CH + t) * D + e, p.g + ((size_t)(t0 + t) * s.heads + h) * s.dim + e);
                }
        } else {
            for (uint32_t t = warp; t < n; t += 8)
                for (uint32_t e = lane; e < s.dim; e += 32) {
                    cp4(b + t * D + e, p.qn + (size_t)(t0 + t) * s.qk + kh * s.dim + e);
                    cp4(b + (CH + t) * D + e, p.kn + (size_t)(t0 + t) * s.qk + kh * s.dim + e);
                    if (!HD) cp4(b + (2 * CH + t) * D + e, p.g + ((size_t)(t0 + t) * s.heads + h) * s.dim + e);
                }
        }
        if (HD && tid < n) cp4(b + 2 * CH * D + tid, p.g + (size_t)(t0 + tid) * s.heads + h);
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
                        if (t < n) run *= b[HD ? 2 * CH * D + t : (2 * CH + t) * D + e];
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
                    if (live) run *= b[HD ? 2 * CH * D + t : (2 * CH + t) * D + e];
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

// The same on tensor cores (bf16 mode, key sizes up to 128): every product with the state is formed from two-term tf32 splits,
// x = hi + lo, as hi hi + hi lo + lo hi, which keeps 22 bits of each factor, with f32 accumulation; the state itself, the
// factors and U stay f32.
//
// Eight warps carry the state: warp = 16 columns x D / PARTS channels, as accumulators of the transposed state (rows = columns
// of S). Those registers are at the same time the B operand of [K'; Q'] S when the eight channels of a step are taken in the
// order 0 2 4 6 1 3 5 7, so the state never leaves them. Eight more warps work one chunk ahead: they fetch q, k, g (three chunks
// ahead) and form the split K', Q', K''.
template <int D, int CB>
struct MmaScanShape {
    static constexpr uint32_t GROUPS = CB / 16, PARTS = 8 / GROUPS, NCH = D / PARTS, NK = NCH / 8;
    static constexpr uint32_t IN = 3 * CH * D, LDF = D + 8, LDU = CB + 8;
    static constexpr uint32_t FAC = 2 * 3 * CH * LDF + D;   // hi then lo of: K' (16 rows), Q' (16), K'' (16); the chunk's decay
    static constexpr uint32_t VTB = CH * CB + 2 * CH * CH;  // v, T, B (four in flight)
    static constexpr uint32_t FLOATS = 3 * IN + 2 * FAC + 4 * VTB + PARTS * 2 * CH * CB + 4 * CH * LDU;
};

// the part of x a tf32 operand holds (x - tf32_hi(x) is exact; of that remainder the tensor core reads the leading bits)
__device__ __forceinline__ float tf32_hi(float x) { return __uint_as_float(__float_as_uint(x) & 0xFFFFE000u); }
__device__ __forceinline__ void mma_tf32(float c[4], const float a[4], float b0, float b1) {
    asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(__float_as_uint(a[0])), "r"(__float_as_uint(a[1])), "r"(__float_as_uint(a[2])), "r"(__float_as_uint(a[3])), "r"(__float_as_uint(b0)),
                   "r"(__float_as_uint(b1)));
}

template <int D, int CB, bool HD>
__global__ void __launch_bounds__(512, 1) delta_scan_mma_kernel(DeltaScan p) {
    using Sh = MmaScanShape<D, CB>;
    constexpr uint32_t LDF = Sh::LDF, LDU = Sh::LDU, NK = Sh::NK, PARTS = Sh::PARTS, TPT = CH * CB / 256;
    extern __shared__ __align__(16) float sm[];
    float *in = sm, *fac = in + 3 * Sh::IN, *vtb = fac + 2 * Sh::FAC, *red = vtb + 4 * Sh::VTB, *X = red + PARTS * 2 * CH * CB, *U = X + CH * LDU, *Uh = U + CH * LDU, *Ul = Uh + CH * LDU;
    const DeltaShape s = p.s;
    const uint32_t h = blockIdx.x, kh = h / (s.heads / s.kv_heads), c0 = blockIdx.y * CB;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    for (uint32_t i = tid; i < Sh::FLOATS; i += 512) sm[i] = 0.0f;  // padding: zero k and q leave padded rows of the state at zero
    __syncthreads();
    pdl_wait();
    pdl_launch();
    store_ring(p, 512);
    const uint32_t ncol = min((uint32_t)CB, s.vdim - c0), chunks = (p.tokens + CH - 1) / CH;
    if (warp >= 8) {  // ---- one chunk ahead ----
        const uint32_t pt = tid - 256, pw = pt >> 5;
        const bool vec = (s.dim & 3) == 0;
        auto fetch = [&](uint32_t chunk) {
            float *b = in + (chunk % 3) * Sh::IN, *bv = vtb + (chunk & 3) * Sh::VTB;
            const uint32_t t0 = chunk * CH, n = min(CH, p.tokens - t0);
            for (uint32_t t = pw; t < n; t += 8) {
                const float *q = p.qn + (size_t)(t0 + t) * s.qk + kh * s.dim, *k = p.kn + (size_t)(t0 + t) * s.qk + kh * s.dim,
                            *g = p.g + ((size_t)(t0 + t) * s.heads + h) * (HD ? 1 : s.dim);
                if (HD && lane == 0) cp4(b + 2 * CH * D + t, g);
                if (vec) {
                    for (uint32_t e = lane * 4; e < s.dim; e += 128) {
                        cp16(b + t * D + e, q + e);
                        cp16(b + (CH + t) * D + e, k + e);
                        if (!HD) cp16(b + (2 * CH + t) * D + e, g + e);
                    }
                } else {
                    for (uint32_t e = lane; e < s.dim; e += 32) {
                        cp4(b + t * D + e, q + e);
                        cp4(b + (CH + t) * D + e, k + e);
                        if (!HD) cp4(b + (2 * CH + t) * D + e, g + e);
                    }
                }
                for (uint32_t e = lane; e < ncol; e += 32) cp4(bv + t * CB + e, p.vn + (size_t)(t0 + t) * s.vd + h * s.vdim + c0 + e);
            }
            if (pt < 128) cp16(bv + CH * CB + 4 * pt, p.tb + ((size_t)chunk * s.heads + h) * 2 * CH * CH + 4 * pt);
            asm volatile("cp.async.commit_group;" ::: "memory");
        };
        auto form = [&](uint32_t chunk) {  // tokens past the end: k = q = 0, no decay
            const float *b = in + (chunk % 3) * Sh::IN;
            float *f = fac + (chunk & 1) * Sh::FAC;
            const uint32_t n = min(CH, p.tokens - chunk * CH);
            auto put = [&](uint32_t row, uint32_t e, float v) {
                const float hi = tf32_hi(v);
                f[row * LDF + e] = hi;
                f[(3 * CH + row) * LDF + e] = v - hi;
            };
            const uint32_t e = pt & 127;  // 128 threads for K' and Q', 128 for K''
            if (e >= D) return;
            float g[CH], k[CH], run = 1.0f;
#pragma unroll
            for (uint32_t t = 0; t < CH; ++t) {
                g[t] = t < n ? b[HD ? 2 * CH * D + t : (2 * CH + t) * D + e] : 1.0f;
                k[t] = t < n ? b[(CH + t) * D + e] : 0.0f;
            }
            if (pt < 128) {
#pragma unroll
                for (uint32_t t = 0; t < CH; ++t) {
                    run *= g[t];
                    put(t, e, k[t] * run);
                    put(CH + t, e, t < n ? b[t * D + e] * run : 0.0f);
                }
            } else {
#pragma unroll
                for (int t = CH - 1; t >= 0; --t) {
                    put(2 * CH + t, e, k[t] * run);
                    run *= g[t];
                }
                f[2 * 3 * CH * LDF + e] = run;
            }
        };
        auto fetch_or_none = [&](uint32_t chunk) {  // (a group per chunk, empty past the end: the waits below count groups)
            if (chunk < chunks) fetch(chunk);
            else asm volatile("cp.async.commit_group;" ::: "memory");
        };
        fetch(0);
        fetch_or_none(1);
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        asm volatile("bar.sync 1, 256;" ::: "memory");
        fetch_or_none(2);
        form(0);
        __syncthreads();
        for (uint32_t chunk = 0; chunk < chunks; ++chunk) {
            if (chunk + 1 < chunks) {
                asm volatile("cp.async.wait_group 1;" ::: "memory");  // chunk + 1 is here
                asm volatile("bar.sync 1, 256;" ::: "memory");
                fetch_or_none(chunk + 3);
                form(chunk + 1);
            }
            __syncthreads();
        }
        return;
    }
    // ---- the state ----
    const uint32_t grp = warp % Sh::GROUPS, part = warp / Sh::GROUPS, g = lane >> 2, q = lane & 3;
    const uint32_t ch0 = part * Sh::NCH, cg = 16 * grp;  // this warp's channels and columns
    float S[NK][4];  // [tile of 8 channels]: columns g and g + 8 x channels 2 q and 2 q + 1
#pragma unroll
    for (uint32_t kt = 0; kt < NK; ++kt)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const uint32_t row = ch0 + 8 * kt + 2 * q + (i & 1), col = c0 + cg + g + 8 * (i >> 1);
            S[kt][i] = (p.pos0 != 0 && row < s.dim && col < s.vdim) ? p.state[((size_t)h * s.dim + row) * s.vdim + col] : 0.0f;
        }
    __syncthreads();
    for (uint32_t chunk = 0; chunk < chunks; ++chunk) {
        const float *fh = fac + (chunk & 1) * Sh::FAC, *fl = fh + 3 * CH * LDF, *cend = fh + 2 * 3 * CH * LDF;
        const float *bv = vtb + (chunk & 3) * Sh::VTB, *bt = bv + CH * CB, *bb = bt + CH * CH;
        const uint32_t t0 = chunk * CH, n = min(CH, p.tokens - t0);
        float big[2][2][4] = {}, small[2][2][4] = {};  // [K', Q'][columns 0-7, 8-15]
#pragma unroll
        for (uint32_t kt = 0; kt < NK; ++kt) {
            float sh[4], sl[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                sh[i] = tf32_hi(S[kt][i]);
                sl[i] = S[kt][i] - sh[i];
            }
#pragma unroll
            for (uint32_t mt = 0; mt < 2; ++mt) {
                const uint32_t at = (mt * CH + g) * LDF + ch0 + 8 * kt + 2 * q;
                const float2 h0 = *reinterpret_cast<const float2 *>(fh + at), h1 = *reinterpret_cast<const float2 *>(fh + at + 8 * LDF);
                const float2 l0 = *reinterpret_cast<const float2 *>(fl + at), l1 = *reinterpret_cast<const float2 *>(fl + at + 8 * LDF);
                const float ah[4] = {h0.x, h1.x, h0.y, h1.y}, al[4] = {l0.x, l1.x, l0.y, l1.y};
#pragma unroll
                for (int nt = 0; nt < 2; ++nt) {
                    mma_tf32(big[mt][nt], ah, sh[2 * nt], sh[2 * nt + 1]);
                    mma_tf32(small[mt][nt], ah, sl[2 * nt], sl[2 * nt + 1]);
                    mma_tf32(small[mt][nt], al, sh[2 * nt], sh[2 * nt + 1]);
                }
            }
        }
#pragma unroll
        for (int mt = 0; mt < 2; ++mt)
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int i = 0; i < 4; i += 2)
                    *reinterpret_cast<float2 *>(red + (part * 2 * CH + mt * CH + g + 4 * i) * CB + cg + 8 * nt + 2 * q) =
                        make_float2(big[mt][nt][i] + small[mt][nt][i], big[mt][nt][i + 1] + small[mt][nt][i + 1]);
        asm volatile("bar.sync 2, 256;" ::: "memory");
        // thread: column uc, tokens ut .. ut + TPT - 1
        const uint32_t uc = tid % CB, ut = tid / CB * TPT;
        float o[TPT];
#pragma unroll
        for (uint32_t i = 0; i < TPT; ++i) {
            const uint32_t t = ut + i;
            float x = bv[t * CB + uc];
            o[i] = 0.0f;
#pragma unroll
            for (uint32_t r = 0; r < PARTS; ++r) {
                x -= red[(r * 2 * CH + t) * CB + uc];
                o[i] += red[(r * 2 * CH + CH + t) * CB + uc];
            }
            X[t * LDU + uc] = t < n ? x : 0.0f;
        }
        asm volatile("bar.sync 2, 256;" ::: "memory");
        {
            float x[CH];
#pragma unroll
            for (uint32_t r = 0; r < CH; ++r) x[r] = X[r * LDU + uc];
#pragma unroll
            for (uint32_t i = 0; i < TPT; ++i) {
                float u = 0.0f;
#pragma unroll
                for (uint32_t r = 0; r < CH; r += 4) {
                    const float4 t = *reinterpret_cast<const float4 *>(bt + (ut + i) * CH + r);
                    u = fmaf(t.x, x[r], fmaf(t.y, x[r + 1], fmaf(t.z, x[r + 2], fmaf(t.w, x[r + 3], u))));
                }
                const float hi = tf32_hi(u);
                Uh[(ut + i) * LDU + uc] = hi;
                Ul[(ut + i) * LDU + uc] = u - hi;
                U[(ut + i) * LDU + uc] = u;
            }
        }
        asm volatile("bar.sync 2, 256;" ::: "memory");
        {  // S <- diag(c) S + K''^T U, transposed: rows = columns of the state
            float uh[2][4], ul[2][4];
#pragma unroll
            for (int ts = 0; ts < 2; ++ts)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const uint32_t at = (8 * ts + q + 4 * (i >> 1)) * LDU + cg + g + 8 * (i & 1);
                    uh[ts][i] = Uh[at];
                    ul[ts][i] = Ul[at];
                }
#pragma unroll
            for (uint32_t kt = 0; kt < NK; ++kt) {
                const float2 c = *reinterpret_cast<const float2 *>(cend + ch0 + 8 * kt + 2 * q);
                S[kt][0] *= c.x;
                S[kt][1] *= c.y;
                S[kt][2] *= c.x;
                S[kt][3] *= c.y;
#pragma unroll
                for (int ts = 0; ts < 2; ++ts) {
                    const uint32_t at = (2 * CH + 8 * ts + q) * LDF + ch0 + 8 * kt + g;
                    const float h0 = fh[at], h1 = fh[at + 4 * LDF], l0 = fl[at], l1 = fl[at + 4 * LDF];
                    mma_tf32(S[kt], uh[ts], l0, l1);
                    mma_tf32(S[kt], ul[ts], h0, h1);
                    mma_tf32(S[kt], uh[ts], h0, h1);
                }
            }
        }
        {
            float u[CH];
#pragma unroll
            for (uint32_t r = 0; r < CH; ++r) u[r] = U[r * LDU + uc];
#pragma unroll
            for (uint32_t i = 0; i < TPT; ++i) {
                const uint32_t t = ut + i;
#pragma unroll
                for (uint32_t r = 0; r < CH; r += 4) {
                    const float4 b = *reinterpret_cast<const float4 *>(bb + t * CH + r);
                    o[i] = fmaf(b.x, u[r], fmaf(b.y, u[r + 1], fmaf(b.z, u[r + 2], fmaf(b.w, u[r + 3], o[i]))));
                }
                if (t < n && uc < ncol) p.o[(size_t)(t0 + t) * s.vd + h * s.vdim + c0 + uc] = o[i];
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (uint32_t kt = 0; kt < NK; ++kt)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const uint32_t row = ch0 + 8 * kt + 2 * q + (i & 1), col = c0 + cg + g + 8 * (i >> 1);
            if (row < s.dim && col < s.vdim) p.state[((size_t)h * s.dim + row) * s.vdim + col] = S[kt][i];
        }
}

// o / rms(o) * w * sigmoid(gate) (SILU: silu(gate)), per head; one warp per (token, head)
template <typename T, bool SILU>
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
    for (uint32_t e = lane; e < vdim; e += 32) {
        const float z = gate[(size_t)t * ldg + h * vdim + e];
        elem_store(out + (size_t)t * ldo + h * vdim + e, x[e] * inv * w[e] * (SILU ? silu_f(z) : sigmoid_f(z)));
    }
}

// ---- one token ---------------------------------------------------------------------------------------------------------
struct DeltaStep {
    DeltaShape s;
    const float *q, *k, *v, *b, *a1, *g1;        // products of this token
    const float *wq, *wk, *wv, *a_log, *dt_bias, *norm;
    const uint16_t *wa2, *wg2;  // null: a1 is the decay's projection with its bias, one per head, and g1 the silu gate's, one per value
    uint32_t ra, rg, lda2, ldg2;
    float *ring, *state, *out;
    const uint32_t *pos;
    float eps;
};
constexpr int STEP_THREADS = 512, STEP_R = 8, STEP_C = 4;  // state kept in registers up to 128 x 128

// eight weights times eight inputs
__device__ __forceinline__ float dot8(const uint4 &q, const float *x, float s) {
    const float4 a = *reinterpret_cast<const float4 *>(x), b = *reinterpret_cast<const float4 *>(x + 4);
    s = fmaf(bf16_lo(q.x), a.x, s);
    s = fmaf(bf16_hi(q.x), a.y, s);
    s = fmaf(bf16_lo(q.y), a.z, s);
    s = fmaf(bf16_hi(q.y), a.w, s);
    s = fmaf(bf16_lo(q.z), b.x, s);
    s = fmaf(bf16_hi(q.z), b.y, s);
    s = fmaf(bf16_lo(q.w), b.z, s);
    return fmaf(bf16_hi(q.w), b.w, s);
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
    // Row i of the head's low-rank factors: the decay's rows, then the gate's. Warp w takes rows w, w + 16, .. in batches of
    // eight; the first batch's weights and the state are asked for ahead of the kernel before this one.
    const uint32_t nrows = p.wa2 ? s.dim + s.vdim : 0u;
    uint4 fw[8];
    auto factor_load = [&](uint32_t r0, uint32_t c) {
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const uint32_t i = r0 + 16 * j;
            const bool decay = i < s.dim;
            fw[j] = (i < nrows && c < (decay ? ra8 : rg8))
                        ? *reinterpret_cast<const uint4 *>(decay ? p.wa2 + (size_t)(h * s.dim + i) * p.lda2 + c : p.wg2 + (size_t)(h * s.vdim + i - s.dim) * p.ldg2 + c)
                        : make_uint4(0, 0, 0, 0);
        }
    };
    factor_load(warp, lane * 8);
    // (the last to write the state was the token before, several kernels ago)
    if (!KEEP)
        for (uint32_t i = tid; i < (s.dim * s.vdim + 31) / 32; i += STEP_THREADS) asm volatile("prefetch.global.L2 [%0];" ::"l"(S + (size_t)i * 32));
    float keep[STEP_R][STEP_C];
    if (KEEP) {
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
    const uint32_t slot = pos % s.taps;
    for (uint32_t i = tid; i < 2 * s.dim + s.vdim; i += STEP_THREADS) {  // (sk follows sq)
        const uint32_t part = i < s.dim ? 0u : (i < 2 * s.dim ? 1u : 2u), c = part < 2 ? kh * s.dim + i - part * s.dim : h * s.vdim + i - 2 * s.dim;
        const float z = silu_f(conv_step(part == 0 ? p.q : (part == 1 ? p.k : p.v), c, part == 0 ? p.wq : (part == 1 ? p.wk : p.wv), cv, slot, part * s.qk + c));
        (part < 2 ? sq[i] : sv[i - 2 * s.dim]) = z;
    }
    __syncthreads();
    // this token's row of the ring (nobody reads it in this step); the heads of a group store the same q and k values
    for (uint32_t i = tid; i < 2 * s.dim + s.vdim; i += STEP_THREADS) {
        const uint32_t ch = i < s.dim ? kh * s.dim + i : (i < 2 * s.dim ? s.qk + kh * s.dim + i - s.dim : 2 * s.qk + h * s.vdim + i - 2 * s.dim);
        const float x = i < s.dim ? p.q[kh * s.dim + i] : (i < 2 * s.dim ? p.k[kh * s.dim + i - s.dim] : p.v[h * s.vdim + i - 2 * s.dim]);
        p.ring[(size_t)slot * cv.channels + ch] = x;
    }
    const float decay = expf(p.a_log[h]);
    if (!p.wa2) {
        for (uint32_t i = tid; i < s.dim; i += STEP_THREADS) sg[i] = expf(-decay * softplus_f(p.a1[h]));
        for (uint32_t i = tid; i < s.vdim; i += STEP_THREADS) gate[i] = silu_f(p.g1[h * s.vdim + i]);
    }
    for (uint32_t r0 = warp; r0 < nrows; r0 += 128) {
        float z[8] = {};
        for (uint32_t c = lane * 8; c < max(ra8, rg8); c += 256) {
            if (r0 != (uint32_t)warp || c != lane * 8) factor_load(r0, c);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const bool dec = r0 + 16 * j < s.dim;
                if (c < (dec ? ra8 : rg8)) z[j] = dot8(fw[j], (dec ? a1 : g1) + c, z[j]);
            }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const uint32_t i = r0 + 16 * j;
            const float v = warp_sum(z[j]);
            if (lane == 0 && i < nrows) {
                if (i < s.dim) sg[i] = expf(-decay * softplus_f(v + p.dt_bias[h * s.dim + i]));
                else gate[i - s.dim] = sigmoid_f(v);
            }
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

class DeltaRule : public Mixer {
  public:
    explicit DeltaRule(bool per_head) : hd_(per_head), name_(per_head ? "delta" : "channel_delta") {}

    bool configure(const brasa::Json &c, uint32_t width, float eps, std::string &err) override {
        if (!read_u32(c, "heads", &s_.heads, err) || !read_u32(c, "kv_heads", &s_.kv_heads, err) || !read_u32(c, "dim", &s_.dim, err) ||
            !read_u32(c, "vdim", &s_.vdim, err) || !read_u32(c, "conv", &s_.taps, err))
            return false;
        if (s_.heads % s_.kv_heads != 0) return err = name_ + ": heads must be a multiple of kv_heads", false;
        if (s_.dim > 256 || s_.vdim > 1024) return err = name_ + ": dim up to 256 and vdim up to 1024", false;
        s_.qk = s_.kv_heads * s_.dim;
        s_.vd = s_.heads * s_.vdim;
        width_ = width;
        eps_ = eps;
        return true;
    }

    int32_t build(Builder &b, const std::string &x) override {
        BRASA_TRY(b.matrix(x + "q", s_.qk, width_, &q_));
        BRASA_TRY(b.matrix(x + "k", s_.qk, width_, &k_));
        BRASA_TRY(b.matrix(x + "v", s_.vd, width_, &v_));
        BRASA_TRY(b.matrix(x + "b", s_.heads, width_, &b_));
        if (hd_) {
            BRASA_TRY(b.matrix(x + "a", s_.heads, width_, &a1_));
            BRASA_TRY(b.matrix(x + "g", s_.vd, width_, &g1_));
        } else {
            BRASA_TRY(b.matrix(x + "a1", 0, width_, &a1_));
            BRASA_TRY(b.matrix(x + "a2", s_.heads * s_.dim, a1_.rows, &a2_));
            BRASA_TRY(b.matrix(x + "g1", 0, width_, &g1_));
            BRASA_TRY(b.matrix(x + "g2", s_.vd, g1_.rows, &g2_));
        }
        outs.resize(1);
        BRASA_TRY(b.matrix(x + "o", width_, s_.vd, &outs[0]));
        BRASA_TRY(b.vector(x + "q.conv", (uint64_t)s_.qk * s_.taps, &wq_));
        BRASA_TRY(b.vector(x + "k.conv", (uint64_t)s_.qk * s_.taps, &wk_));
        BRASA_TRY(b.vector(x + "v.conv", (uint64_t)s_.vd * s_.taps, &wv_));
        BRASA_TRY(b.vector(x + "A_log", s_.heads, &a_log_));
        BRASA_TRY(b.vector(x + "dt_bias", (uint64_t)s_.heads * (hd_ ? 1 : s_.dim), &dt_bias_));
        BRASA_TRY(b.vector(x + "norm", s_.vdim, &norm_));
        BRASA_TRY(b.get(Builder::STATE, 4ull * s_.taps * (2 * s_.qk + s_.vd), (void **)&ring_));
        BRASA_TRY(b.get(Builder::STATE, 4ull * s_.heads * s_.dim * s_.vdim, (void **)&state_));
        lay_out(b.limits.max_tokens, b.f32);
        return BRASA_OK;
    }

    uint64_t scratch_bytes() const override { return at_.total; }

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
        if (hd_) {
            add(a1_, at_.z, ldz_, false);
            out.back().p.bias = dt_bias_;
            add(g1_, at_.gate, ldv_, false);
        } else {
            add(a1_, at_.a1, lda_, true);  // inputs of a product: bf16 where products take bf16
            add(g1_, at_.g1, ldg_, true);
        }
    }

    int32_t mix(const Run &r) override {
        brasa_ctx *ctx = r.cmd->ctx;
        auto f = [&](uint64_t at) { return (float *)(r.scratch + at); };
        if (r.dev_pos) {
            DeltaStep p{s_, f(at_.q), f(at_.k), f(at_.v), f(at_.b), hd_ ? f(at_.z) : f(at_.a1), hd_ ? f(at_.gate) : f(at_.g1), wq_, wk_, wv_, a_log_, dt_bias_, norm_,
                        a2_.p, g2_.p, a2_.cols, g2_.cols, a2_.ld, g2_.ld, ring_, state_, (float *)r.out[0], r.dev_pos, eps_};
            const size_t smem = step_smem(s_, a2_.cols, g2_.cols);
            const bool keep = s_.dim <= 16 * STEP_R && s_.vdim <= 32 * STEP_C;
            const void *fn = keep ? (const void *)delta_step_kernel<true> : (const void *)delta_step_kernel<false>;
            BRASA_TRY(brasa_smem_optin(ctx, fn, smem));
            if (keep) BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_step_kernel<true>, dim3(s_.heads), dim3(STEP_THREADS), smem, p));
            else BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_step_kernel<false>, dim3(s_.heads), dim3(STEP_THREADS), smem, p));
            return brasa_post_launch(r.cmd, "delta_step");
        }
        if (!hd_) {  // the second factors of the decay's and the gate's projections
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
        }
        const uint32_t channels = 2 * s_.qk + s_.vd;
        DeltaChunk cp{s_, ConvView{ring_, channels, s_.taps, r.pos0}, f(at_.q), f(at_.k), f(at_.v), f(at_.b), f(at_.z), ldqk_, ldv_, ldb_, ldz_, r.tokens, wq_, wk_, wv_, a_log_,
                      f(at_.qn), f(at_.kn), f(at_.vn), f(at_.g), f(at_.tb)};
        if (hd_) BRASA_TRY(factors_any<true>(r.cmd, cp));
        else BRASA_TRY(factors_any<false>(r.cmd, cp));
        DeltaScan sp{s_, f(at_.qn), f(at_.kn), f(at_.vn), f(at_.g), f(at_.tb), f(at_.q), f(at_.k), f(at_.v), ldqk_, ldv_, ring_, state_, f(at_.o), r.tokens, r.pos0};
        if (hd_) BRASA_TRY(scan<true>(r.cmd, sp, r.f32));
        else BRASA_TRY(scan<false>(r.cmd, sp, r.f32));
        const uint32_t blocks = (r.tokens * s_.heads + 7) / 8;
        auto out = [&](auto kernel, auto *dst) {
            return brasa_launch_dependent(ctx, kernel, dim3(blocks), dim3(256), 0, f(at_.o), f(at_.gate), ldv_, norm_, dst, r.ldo[0], s_.heads, s_.vdim, r.tokens, eps_);
        };
        if (r.f32) BRASA_CUDA(ctx, hd_ ? out(delta_out_kernel<float, true>, (float *)r.out[0]) : out(delta_out_kernel<float, false>, (float *)r.out[0]));
        else BRASA_CUDA(ctx, hd_ ? out(delta_out_kernel<__nv_bfloat16, true>, (__nv_bfloat16 *)r.out[0]) : out(delta_out_kernel<__nv_bfloat16, false>, (__nv_bfloat16 *)r.out[0]));
        return brasa_post_launch(r.cmd, "delta_out");
    }

  private:
    template <bool HD>
    int32_t factors_any(brasa_cmd *cmd, const DeltaChunk &p) {
        if (s_.dim <= 64) return factors<2, HD>(cmd, p);
        if (s_.dim <= 128) return factors<4, HD>(cmd, p);
        return factors<8, HD>(cmd, p);
    }
    template <int E, bool HD>
    int32_t factors(brasa_cmd *cmd, const DeltaChunk &p) {
        brasa_ctx *ctx = cmd->ctx;
        const size_t smem = 3ull * CH * 32 * E * 4;
        BRASA_TRY(brasa_smem_optin(ctx, (const void *)delta_chunk_kernel<E, HD>, std::max<size_t>(smem, 48 * 1024)));
        BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_chunk_kernel<E, HD>, dim3((p.tokens + CH - 1) / CH, s_.heads), dim3(256), smem, p));
        return brasa_post_launch(cmd, "delta_chunk");
    }
    template <int D, int CB, bool HD>
    int32_t scan_as(brasa_cmd *cmd, const DeltaScan &p) {
        brasa_ctx *ctx = cmd->ctx;
        const size_t smem = (size_t)ScanShape<D, CB>::FLOATS * 4;
        BRASA_TRY(brasa_smem_optin(ctx, (const void *)delta_scan_kernel<D, CB, HD>, smem));
        BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_scan_kernel<D, CB, HD>, dim3(s_.heads, (s_.vdim + CB - 1) / CB), dim3(256), smem, p));
        return brasa_post_launch(cmd, "delta_scan");
    }
    template <int D, int CB, bool HD>
    int32_t scan_mma(brasa_cmd *cmd, const DeltaScan &p) {
        brasa_ctx *ctx = cmd->ctx;
        const size_t smem = (size_t)MmaScanShape<D, CB>::FLOATS * 4;
        BRASA_TRY(brasa_smem_optin(ctx, (const void *)delta_scan_mma_kernel<D, CB, HD>, smem));
        BRASA_CUDA(ctx, brasa_launch_dependent(ctx, delta_scan_mma_kernel<D, CB, HD>, dim3(s_.heads, (s_.vdim + CB - 1) / CB), dim3(512), smem, p));
        return brasa_post_launch(cmd, "delta_scan_mma");
    }
    template <bool HD>
    int32_t scan(brasa_cmd *cmd, const DeltaScan &p, bool f32) {
        // wide blocks when they still cover most of the SMs
        const bool wide = s_.heads * ((s_.vdim + 31) / 32) * 5 >= (uint32_t)cmd->ctx->sm_count * 4;
        if (!f32 && s_.dim <= 64) return wide ? scan_mma<64, 32, HD>(cmd, p) : scan_mma<64, 16, HD>(cmd, p);
        if (!f32 && s_.dim <= 128) return wide ? scan_mma<128, 32, HD>(cmd, p) : scan_mma<128, 16, HD>(cmd, p);
        if (s_.dim <= 64) return wide ? scan_as<64, 32, HD>(cmd, p) : scan_as<64, 16, HD>(cmd, p);
        if (s_.dim <= 128) return wide ? scan_as<128, 32, HD>(cmd, p) : scan_as<128, 16, HD>(cmd, p);
        return scan_as<256, 16, HD>(cmd, p);
    }

    void lay_out(uint64_t t, bool f32) {
        ldqk_ = up8(s_.qk);
        ldv_ = up8(s_.vd);
        ldb_ = up8(s_.heads);
        lda_ = up8(a1_.rows);
        ldg_ = up8(g1_.rows);
        ldz_ = up8(s_.heads * (hd_ ? 1 : s_.dim));
        (void)f32;
        Carver c;
        at_.q = c.take(4 * t * ldqk_);
        at_.k = c.take(4 * t * ldqk_);
        at_.v = c.take(4 * t * ldv_);
        at_.b = c.take(4 * t * ldb_);
        at_.a1 = c.take(hd_ ? 0 : 4 * t * lda_);
        at_.g1 = c.take(hd_ ? 0 : 4 * t * ldg_);
        at_.z = c.take(4 * t * ldz_);
        at_.gate = c.take(4 * t * ldv_);
        at_.qn = c.take(4 * t * s_.qk);
        at_.kn = c.take(4 * t * s_.qk);
        at_.vn = c.take(4 * t * s_.vd);
        at_.g = c.take(4 * t * s_.heads * (hd_ ? 1 : s_.dim));
        at_.tb = c.take(4ull * ((t + CH - 1) / CH) * s_.heads * 2 * CH * CH);
        at_.o = c.take(4 * t * s_.vd);
        at_.total = c.at;
    }

    const bool hd_;  // one decay per head
    const std::string name_;
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

std::unique_ptr<Mixer> make_channel_delta() { return std::unique_ptr<Mixer>(new DeltaRule(false)); }
std::unique_ptr<Mixer> make_delta() { return std::unique_ptr<Mixer>(new DeltaRule(true)); }

}  // namespace brasa_stack
