// Products with bfloat16 weights: a persistent tcgen05 GEMM for many tokens, an f32 form of it, and a weight-streaming GEMV
// for one token. Several products that a layer runs side by side go into one launch (linear.h).
#include <string.h>

#include "linear.h"
#include "tc_device.cuh"

using namespace brasa_dev;

namespace {

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float activate(float v, int act) {
    if (act == LINEAR_ACT_RELU2) {
        v = fmaxf(v, 0.0f);
        v *= v;
    } else if (act == LINEAR_ACT_GELU_TANH) {
        v = v / (1.0f + expf(-1.5957691216057308f * fmaf(0.044715f * v * v, v, v)));  // 0.5 (1 + tanh(u)) = 1 / (1 + exp(-2 u))
    }
    return v;
}
// the epilogue behind the sum and its bias, up to the residual
__device__ __forceinline__ float finish(float v, int act, float scale, float cap) {
    v = activate(v, act) * scale;
    return cap > 0.0f ? cap * tanhf(v / cap) : v;
}
__device__ __forceinline__ float mul_at(const uint16_t *mul, uint32_t ldm, uint32_t id, uint32_t r) {
    return __uint_as_float((uint32_t)mul[(size_t)id * ldm + r] << 16);
}

// ---- f32: inputs f32 (or bf16), weights bf16, f32 FMA. Block 16 x 16 threads, each 4 tokens x 4 rows. -----------------
struct SimtParams {
    LinearProblem p[LINEAR_MAX];
    uint32_t tile_end[LINEAR_MAX];  // 64 x 64 output tiles of problems 0..i, cumulative
    uint32_t n;
};
constexpr int TM = 64, TN = 64, TK = 32;

__global__ void __launch_bounds__(256) linear_f32_kernel(const __grid_constant__ SimtParams sp) {
    __shared__ float xs[TM][TK + 1], ws[TN][TK + 1];
    uint32_t pi = 0;
    while (pi + 1 < sp.n && blockIdx.x >= sp.tile_end[pi]) ++pi;
    const LinearProblem &p = sp.p[pi];
    const uint32_t tile = blockIdx.x - (pi ? sp.tile_end[pi - 1] : 0u), row_tiles = (p.rows + TN - 1) / TN;
    const uint32_t row0 = tile % row_tiles * TN, tok0 = tile / row_tiles * TM;
    const int t = threadIdx.x, ty = t >> 4, tx = t & 15;
    float acc[4][4] = {};
    for (int s = 0; s < 2; ++s) {
        const LinearSeg &g = p.seg[s];
        const float *x = static_cast<const float *>(g.x);
        for (uint32_t k0 = 0; k0 < g.cols; k0 += TK) {
            for (int i = t; i < TM * TK; i += 256) {
                const uint32_t r = i / TK, c = k0 + i % TK;
                xs[r][i % TK] = (tok0 + r < p.tokens && c < g.cols) ? x[(size_t)(tok0 + r) * g.ldx + c] : 0.0f;
                ws[r][i % TK] = (row0 + r < p.rows && c < g.cols) ? __uint_as_float((uint32_t)g.w[(size_t)(row0 + r) * g.ldw + c] << 16) : 0.0f;
            }
            __syncthreads();
#pragma unroll 8
            for (int k = 0; k < TK; ++k) {
                float xv[4], wv[4];
                for (int i = 0; i < 4; ++i) {
                    xv[i] = xs[ty + 16 * i][k];
                    wv[i] = ws[tx + 16 * i][k];
                }
                for (int i = 0; i < 4; ++i)
                    for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
            }
            __syncthreads();
        }
    }
    const bool glu = p.act == LINEAR_ACT_SWIGLU;  // tile rows 0-31 are gate rows, 32-63 their up rows
    for (int i = 0; i < 4; ++i)
        for (int j = 0; j < (glu ? 2 : 4); ++j) {
            const uint32_t tok = tok0 + ty + 16 * i, r = (glu ? row0 / 2 : row0) + tx + 16 * j;
            if (tok >= p.tokens || r >= (glu ? p.rows / 2 : p.rows)) continue;
            const size_t at = (size_t)tok * p.ldy + r;
            float v = glu ? silu_f(acc[i][j]) * acc[i][j + 2] : finish(acc[i][j] + (p.bias ? p.bias[r] : 0.0f), p.act, p.scale, p.cap);
            if (p.mul) v *= mul_at(p.mul, p.ldm, p.mul_ids[tok], r);
            if (p.resid) v += p.resid[at];
            if (p.y_bf16) static_cast<__nv_bfloat16 *>(p.y)[at] = __float2bfloat16_rn(v);
            else static_cast<float *>(p.y)[at] = v;
        }
}

// ---- one token: GEMV ---------------------------------------------------------------------------------------------------
// One block of 32 warps per SM. S warps share a row (K split), a row's weights are read 16 bytes per lane; the block's input
// vectors sit in shared memory in two planes (elements 0-3 and 4-7 of every eight), so that a lane's eight values are two
// conflict-free 16-byte loads. The first weights are asked for before the dependency wait: they never change.
struct GemvDevProblem {
    const uint16_t *w[2];
    uint32_t ldw[2], cols8[2], xoff[2];  // cols8: columns rounded up to eight (padding is zero on both sides)
    uint32_t rows;
    float *y;
    const float *bias, *resid;
    int act;
    float scale, cap;
    const uint16_t *mul;
    const uint32_t *mul_id;
    uint32_t ldm;
};
struct GemvDevParams {
    GemvDevProblem p[LINEAR_MAX];
    uint32_t row_end[LINEAR_MAX];
    uint32_t n, total_rows;
    const float *x, *y, *wy;
    float *x_out;
    int norm;
    uint32_t width, nin;
    float eps;
    const float *w[2], *b[2], *v[2], *vw[2];
    float vscale[2];
    uint32_t len[2], off[2], parts[2], x_floats;
    bool gated;
};
constexpr int GV_WARPS = 32, GV_UNROLL = 4;

__device__ __forceinline__ uint32_t gv_plane(uint32_t e, uint32_t half) { return ((e >> 2) & 1) * half + ((e >> 3) << 2) + (e & 3); }

__device__ __forceinline__ float block_sum_1024(float v, float *red) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    v = red[threadIdx.x & 31];
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    __syncthreads();
    return v;
}

// IN: what the input is formed from.
enum { IN_VECTORS, IN_STREAM, IN_LAYER_NORM };
template <int S, int IN>
__global__ void __launch_bounds__(32 * GV_WARPS, 1) linear_gemv_kernel(const __grid_constant__ GemvDevParams gp) {
    extern __shared__ __align__(16) float xs[];
    __shared__ float red[32], part[2][GV_WARPS];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    constexpr uint32_t TEAMS = GV_WARPS / S;
    const uint32_t team = blockIdx.x * TEAMS + warp / S, teams = gridDim.x * TEAMS, sub = warp % S;
    const uint32_t half = gp.x_floats / 2;
    // A warp's work is a list of batches of up to GV_UNROLL x 16 bytes per lane: along a row's first segment, its second, the
    // team's next row, .. The next batch's weights are in flight while this one is multiplied.
    struct Cursor {
        uint32_t row, pi, r, seg, c0;
    };
    auto place = [&](Cursor &c) {  // problem and row of c.row
        c.pi = 0;
        while (c.pi + 1 < gp.n && c.row >= gp.row_end[c.pi]) ++c.pi;
        c.r = c.row - (c.pi ? gp.row_end[c.pi - 1] : 0u);
    };
    auto load = [&](const Cursor &c, uint4 *q) {
        const GemvDevProblem &p = gp.p[c.pi];
        const uint32_t cols = p.cols8[c.seg];
        const uint16_t *w = p.w[c.seg] + (size_t)c.r * p.ldw[c.seg];
#pragma unroll
        for (int u = 0; u < GV_UNROLL; ++u) {
            const uint32_t k = c.c0 + (sub * 32 + lane) * 8 + u * 256 * S;
            q[u] = k < cols ? __ldcs(reinterpret_cast<const uint4 *>(w + k)) : make_uint4(0, 0, 0, 0);
        }
    };
    auto advance = [&](Cursor &c) {  // false at the end; a new row has seg == 0 and c0 == 0
        c.c0 += GV_UNROLL * 256 * S;
        if (c.c0 < gp.p[c.pi].cols8[c.seg]) return true;
        c.c0 = 0;
        if (c.seg == 0 && gp.p[c.pi].cols8[1]) {
            c.seg = 1;
            return true;
        }
        c.seg = 0;
        c.row += teams;
        if (c.row >= gp.total_rows) return false;
        place(c);
        return true;
    };
    Cursor cur{team, 0, 0, 0, 0};
    bool more = team < gp.total_rows;
    uint4 q[GV_UNROLL];
    if (more) {
        place(cur);
        load(cur, q);
    }
    // ---- the input vectors ----
    // Up to GV_KEEP values of the residual stream per thread stay in registers, with the constants asked for ahead of the wait.
    constexpr uint32_t GV_KEEP = 4, GV_T = 32 * GV_WARPS;
    constexpr bool LN = IN == IN_LAYER_NORM;
    const bool keep = gp.width <= GV_KEEP * GV_T;
    float xk[GV_KEEP], yk[GV_KEEP], wk[GV_KEEP], bk[GV_KEEP];
    if (IN != IN_VECTORS && keep)
#pragma unroll
        for (uint32_t j = 0; j < GV_KEEP; ++j) {
            const uint32_t i = tid + GV_T * j;
            const float *b = LN ? gp.b[0] : (gp.y ? gp.wy : nullptr);
            wk[j] = (LN || gp.norm == GEMV_RMS_NORM) && i < gp.width ? gp.w[0][i] : 1.0f;
            bk[j] = b && i < gp.width ? b[i] : 0.0f;
        }
    pdl_wait();
    pdl_launch();
    for (uint32_t k = 0; k < gp.nin; ++k)  // padding
        if (tid < 8 && (gp.len[k] & 7) && gp.len[k] / 8 * 8 + tid >= gp.len[k]) xs[gv_plane(gp.off[k] + gp.len[k] / 8 * 8 + tid, half)] = 0.0f;
    if (IN != IN_VECTORS && keep) {
        float s = 0.0f;
#pragma unroll
        for (uint32_t j = 0; j < GV_KEEP; ++j) {
            const uint32_t i = tid + GV_T * j;
            xk[j] = i < gp.width ? gp.x[i] : 0.0f;
            yk[j] = !LN && gp.y && i < gp.width ? gp.y[i] : 0.0f;
        }
        if (LN) {
#pragma unroll
            for (uint32_t j = 0; j < GV_KEEP; ++j) s += xk[j];
            const float mean = block_sum_1024(s, red) / (float)gp.width;
            s = 0.0f;
#pragma unroll
            for (uint32_t j = 0; j < GV_KEEP; ++j) {
                xk[j] -= mean;
                if (tid + GV_T * j < gp.width) s = fmaf(xk[j], xk[j], s);
            }
            const float inv = 1.0f / sqrtf(block_sum_1024(s, red) / (float)gp.width + gp.eps);
#pragma unroll
            for (uint32_t j = 0; j < GV_KEEP; ++j) {
                const uint32_t i = tid + GV_T * j;
                if (i < gp.width) {
                    xs[gv_plane(gp.off[0] + i, half)] = fmaf(xk[j] * inv, wk[j], bk[j]);
                    if (gp.nin > 1) xs[gv_plane(gp.off[1] + i, half)] = fmaf(xk[j] * inv, gp.w[1][i], gp.b[1][i]);
                }
            }
        } else {
            if (gp.y) {
#pragma unroll
                for (uint32_t j = 0; j < GV_KEEP; ++j) s = fmaf(yk[j], yk[j], s);
                const float sy = 1.0f / sqrtf(block_sum_1024(s, red) / (float)gp.width + gp.eps);
                s = 0.0f;
#pragma unroll
                for (uint32_t j = 0; j < GV_KEEP; ++j) {
                    const uint32_t i = tid + GV_T * j;
                    xk[j] = fmaf(yk[j] * sy, bk[j], xk[j]);
                    if (blockIdx.x == 0 && gp.x_out && i < gp.width) gp.x_out[i] = xk[j];
                }
            }
            float inv = 1.0f;
            if (gp.norm == GEMV_RMS_NORM) {
#pragma unroll
                for (uint32_t j = 0; j < GV_KEEP; ++j) s = fmaf(xk[j], xk[j], s);
                inv = 1.0f / sqrtf(block_sum_1024(s, red) / (float)gp.width + gp.eps);
            }
#pragma unroll
            for (uint32_t j = 0; j < GV_KEEP; ++j)
                if (tid + GV_T * j < gp.width) xs[gv_plane(gp.off[0] + tid + GV_T * j, half)] = xk[j] * inv * wk[j];
        }
    } else if (IN != IN_VECTORS) {
        // a wider stream: its values in shared memory meanwhile; every thread keeps to its own elements
        float s = 0.0f, sy = 0.0f;
        if (!LN && gp.y) {
            for (uint32_t i = tid; i < gp.width; i += GV_T) s = fmaf(gp.y[i], gp.y[i], s);
            sy = 1.0f / sqrtf(block_sum_1024(s, red) / (float)gp.width + gp.eps);
        }
        s = 0.0f;
        for (uint32_t i = tid; i < gp.width; i += GV_T) {
            float v = gp.x[i];
            if (!LN && gp.y) {
                v = fmaf(gp.y[i] * sy, gp.wy[i], v);
                if (blockIdx.x == 0 && gp.x_out) gp.x_out[i] = v;
            }
            xs[gv_plane(gp.off[0] + i, half)] = v;
            s += LN ? v : v * v;
        }
        if (LN) {
            const float mean = block_sum_1024(s, red) / (float)gp.width;
            s = 0.0f;
            for (uint32_t i = tid; i < gp.width; i += GV_T) {
                const float d = xs[gv_plane(gp.off[0] + i, half)] - mean;
                s = fmaf(d, d, s);
            }
            const float inv = 1.0f / sqrtf(block_sum_1024(s, red) / (float)gp.width + gp.eps);
            for (uint32_t i = tid; i < gp.width; i += GV_T) {
                const float z = (xs[gv_plane(gp.off[0] + i, half)] - mean) * inv;
                xs[gv_plane(gp.off[0] + i, half)] = fmaf(z, gp.w[0][i], gp.b[0][i]);
                if (gp.nin > 1) xs[gv_plane(gp.off[1] + i, half)] = fmaf(z, gp.w[1][i], gp.b[1][i]);
            }
        } else if (gp.norm == GEMV_RMS_NORM) {
            const float inv = 1.0f / sqrtf(block_sum_1024(s, red) / (float)gp.width + gp.eps);
            for (uint32_t i = tid; i < gp.width; i += GV_T) xs[gv_plane(gp.off[0] + i, half)] *= inv * gp.w[0][i];
        }
    } else {
        // (loads go out several at a time, ahead of the stores to shared memory)
        constexpr uint32_t AT = 4;
        for (uint32_t k = 0; k < gp.nin; ++k) {
            if (gp.gated && k == 0) {
                for (uint32_t i0 = tid; i0 < gp.len[0]; i0 += AT * GV_T) {
                    float g[AT], u[AT];
#pragma unroll
                    for (uint32_t j = 0; j < AT; ++j) {
                        const uint32_t i = i0 + GV_T * j;
                        const float *src = gp.v[0] + (size_t)(i >> 5) * 64 + (i & 31);
                        g[j] = i < gp.len[0] ? src[0] : 0.0f;
                        u[j] = i < gp.len[0] ? src[32] : 0.0f;
                    }
#pragma unroll
                    for (uint32_t j = 0; j < AT; ++j)
                        if (i0 + GV_T * j < gp.len[0]) xs[gv_plane(gp.off[0] + i0 + GV_T * j, half)] = silu_f(g[j]) * u[j];
                }
            } else if (gp.parts[k]) {
                // a warp takes parts warp, warp + 32, .. where there are many; otherwise a part is the block's
                const uint32_t n = gp.len[k] / gp.parts[k];
                if (gp.parts[k] >= GV_WARPS / 2) {
                    for (uint32_t part = warp; part < gp.parts[k]; part += GV_WARPS) {
                        float s = 0.0f;
                        for (uint32_t i = lane; i < n; i += 32) s = fmaf(gp.v[k][part * n + i], gp.v[k][part * n + i], s);
#pragma unroll
                        for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
                        const float inv = gp.vscale[k] / sqrtf(s / (float)n + gp.eps);
                        for (uint32_t i = lane; i < n; i += 32) xs[gv_plane(gp.off[k] + part * n + i, half)] = gp.v[k][part * n + i] * inv * gp.vw[k][part * n + i];
                    }
                } else {
                    for (uint32_t part = 0; part < gp.parts[k]; ++part) {
                        float s = 0.0f;
                        for (uint32_t i0 = tid; i0 < n; i0 += AT * GV_T) {
                            float v[AT], w[AT];
#pragma unroll
                            for (uint32_t j = 0; j < AT; ++j) {
                                const uint32_t i = i0 + GV_T * j;
                                v[j] = i < n ? gp.v[k][part * n + i] : 0.0f;
                                w[j] = i < n ? gp.vw[k][part * n + i] : 0.0f;
                            }
#pragma unroll
                            for (uint32_t j = 0; j < AT; ++j) {
                                if (i0 + GV_T * j < n) xs[gv_plane(gp.off[k] + part * n + i0 + GV_T * j, half)] = v[j] * w[j];
                                s = fmaf(v[j], v[j], s);
                            }
                        }
                        const float inv = gp.vscale[k] / sqrtf(block_sum_1024(s, red) / (float)n + gp.eps);
                        for (uint32_t i = tid; i < n; i += GV_T) xs[gv_plane(gp.off[k] + part * n + i, half)] *= inv;
                    }
                }
            } else {
                for (uint32_t i0 = tid; i0 < gp.len[k]; i0 += AT * GV_T) {
                    float v[AT];
#pragma unroll
                    for (uint32_t j = 0; j < AT; ++j) v[j] = i0 + GV_T * j < gp.len[k] ? gp.v[k][i0 + GV_T * j] : 0.0f;
#pragma unroll
                    for (uint32_t j = 0; j < AT; ++j)
                        if (i0 + GV_T * j < gp.len[k]) xs[gv_plane(gp.off[k] + i0 + GV_T * j, half)] = v[j];
                }
            }
        }
    }
    __syncthreads();
    // ---- batches ----
    float acc = 0.0f;
    uint32_t parity = 0;
    while (more) {
        Cursor nxt = cur;
        const bool go_on = advance(nxt);
        uint4 qn[GV_UNROLL];
        if (go_on) load(nxt, qn);
        const GemvDevProblem &p = gp.p[cur.pi];
        const float *x = xs + (p.xoff[cur.seg] >> 1);
        const uint32_t cols = p.cols8[cur.seg];
#pragma unroll
        for (int u = 0; u < GV_UNROLL; ++u) {
            const uint32_t c = cur.c0 + (sub * 32 + lane) * 8 + u * 256 * S;
            if (c < cols) {
                const float4 a = *reinterpret_cast<const float4 *>(x + (c >> 1)), b = *reinterpret_cast<const float4 *>(x + half + (c >> 1));
                acc = fmaf(bf16_lo(q[u].x), a.x, acc);
                acc = fmaf(bf16_hi(q[u].x), a.y, acc);
                acc = fmaf(bf16_lo(q[u].y), a.z, acc);
                acc = fmaf(bf16_hi(q[u].y), a.w, acc);
                acc = fmaf(bf16_lo(q[u].z), b.x, acc);
                acc = fmaf(bf16_hi(q[u].z), b.y, acc);
                acc = fmaf(bf16_lo(q[u].w), b.z, acc);
                acc = fmaf(bf16_hi(q[u].w), b.w, acc);
            }
        }
        if (!go_on || (nxt.seg == 0 && nxt.c0 == 0)) {  // the row is complete
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
            if (S > 1) {  // (the warps of a team walk the same batches)
                if (lane == 0) part[parity][warp] = acc;
                asm volatile("bar.sync %0, %1;" ::"r"(warp / S), "r"(32 * S) : "memory");
                if (sub == 0 && lane == 0)
                    for (int k = 1; k < S; ++k) acc += part[parity][warp + k];
                parity ^= 1;
            }
            if (sub == 0 && lane == 0) {
                float v = finish(acc + (p.bias ? p.bias[cur.r] : 0.0f), p.act, p.scale, p.cap);
                if (p.mul) v *= mul_at(p.mul, p.ldm, *p.mul_id, cur.r);
                if (p.resid) v += p.resid[cur.r];
                p.y[cur.r] = v;
            }
            acc = 0.0f;
        }
        more = go_on;
        cur = nxt;
#pragma unroll
        for (int u = 0; u < GV_UNROLL; ++u) q[u] = qn[u];
    }
}

// ---- many tokens: tcgen05 ----------------------------------------------------------------------------------------------
// Persistent, one CTA per SM, tiles of 128 tokens x BN weight rows dealt out in order over all problems. Warp 0 (one lane):
// TMA of X and W tiles (128-byte swizzle; rows, tokens and columns past the end read as zeros) into a ring of stages of 64
// columns. Warp 1 (one lane): tcgen05.mma, M = 128 tokens, N = BN rows, into one of two accumulators in tensor memory.
// Warps 4-7: epilogue of the finished accumulator while the next tile is computed: 32 x 32 blocks are turned around in
// shared memory so that stores (and the residual's loads) run along the rows of Y.
// Every wait is bounded: a wait that runs out raises the context's status word, every role leaves, tensor memory is freed.
constexpr uint32_t BM = 128, BK = 64, TC_WAIT = 1u << 22;
constexpr uint32_t EPI_LD = 36, EPI_BYTES = 4 * 32 * EPI_LD * 4;

struct TcProblem {
    uint32_t rows, tokens, tok_tiles, stages0, stages;  // stages0: K stages of the first segment
    void *y;
    uint32_t ldy, y_bf16;
    const float *bias, *resid;
    int act;
    float scale, cap;
    const uint16_t *mul;
    const uint32_t *mul_ids;
    uint32_t ldm;
};
struct TcParams {
    CUtensorMap x[LINEAR_MAX][2], w[LINEAR_MAX][2];
    TcProblem p[LINEAR_MAX];
    uint32_t tile_end[LINEAR_MAX];
    uint32_t n, tiles;
    uint32_t *status;
};

template <int BN>
struct TcShape {
    static constexpr uint32_t STAGE = BM * BK * 2 + BN * BK * 2;
    static constexpr uint32_t NS = BN == 256 ? 4 : (BN == 128 ? 6 : 8);
    static constexpr size_t SMEM = (size_t)NS * STAGE + EPI_BYTES + 1024;
};

// One warp's 32 tokens (from tok on) of a finished accumulator, ncol columns, by way of the warp's stage of shared memory. A kind
// of its own for each of: bias, squared relu, scale and residual; gated rows; gelu times a factor; everything else. (What a kind
// does not have is not in its loop, whose loads and stores can then overlap.)
enum { EPI_PLAIN, EPI_GATED, EPI_GELU_MUL, EPI_ANY };
template <int EPI>
__device__ __forceinline__ void tile_out(const TcProblem &p, uint32_t acc, float *stage, uint32_t row0, uint32_t ncol, uint32_t tok, int lane) {
    const uint32_t tr = lane >> 3, tc = (lane & 7) * 4;  // this lane's row and columns of the turned block
    const uint32_t out_rows = EPI == EPI_GATED ? p.rows / 2 : p.rows;
    for (uint32_t c0 = 0; c0 < ncol; c0 += EPI == EPI_GATED ? 64 : 32) {
        uint32_t v[32];
        tc_ld32(acc + c0, v);
        if (EPI == EPI_GATED) {
            uint32_t u[32];
            tc_ld32(acc + c0 + 32, u);
#pragma unroll
            for (int e = 0; e < 32; ++e) {
                const float g = __uint_as_float(v[e]);
                v[e] = __float_as_uint(__fdividef(g, 1.0f + __expf(-g)) * __uint_as_float(u[e]));
            }
        }
#pragma unroll
        for (int g = 0; g < 8; ++g)
            *reinterpret_cast<float4 *>(stage + lane * EPI_LD + 4 * g) =
                make_float4(__uint_as_float(v[4 * g]), __uint_as_float(v[4 * g + 1]), __uint_as_float(v[4 * g + 2]), __uint_as_float(v[4 * g + 3]));
        __syncwarp();
        const uint32_t r = (EPI == EPI_GATED ? (row0 + c0) / 2 : row0 + c0) + tc;
        float bias[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) bias[e] = (EPI != EPI_GATED && EPI != EPI_GELU_MUL && p.bias && r + e < out_rows) ? p.bias[r + e] : 0.0f;
        const bool vec = r + 4 <= out_rows && (p.ldy & 3) == 0;
        uint16_t f[8][4];  // the factors, all asked for at once
        if (EPI == EPI_GELU_MUL) {
            uint32_t id[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) id[i] = tok + 4 * i + tr < p.tokens ? p.mul_ids[tok + 4 * i + tr] : 0u;
#pragma unroll
            for (int i = 0; i < 8; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) f[i][e] = tok + 4 * i + tr < p.tokens && r + e < out_rows ? p.mul[(size_t)id[i] * p.ldm + r + e] : (uint16_t)0;
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const uint32_t t = tok + 4 * i + tr;
            if (t < p.tokens && r < out_rows) {
                const float4 a = *reinterpret_cast<const float4 *>(stage + (4 * i + tr) * EPI_LD + tc);
                float o[4] = {a.x, a.y, a.z, a.w};
                if (EPI == EPI_PLAIN) {
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        o[e] += bias[e];
                        if (p.act == LINEAR_ACT_RELU2) {
                            o[e] = fmaxf(o[e], 0.0f);
                            o[e] *= o[e];
                        }
                        o[e] *= p.scale;
                    }
                }
                if (EPI == EPI_GELU_MUL) {
#pragma unroll
                    for (int e = 0; e < 4; ++e)
                        o[e] = __fdividef(o[e], 1.0f + __expf(-1.5957691216057308f * fmaf(0.044715f * o[e] * o[e], o[e], o[e]))) * __uint_as_float((uint32_t)f[i][e] << 16);
                }
                if (EPI == EPI_ANY) {
#pragma unroll
                    for (int e = 0; e < 4; ++e) o[e] = finish(o[e] + bias[e], p.act, p.scale, p.cap);
                    if (p.mul)
                        for (int e = 0; e < 4 && r + e < out_rows; ++e) o[e] *= mul_at(p.mul, p.ldm, p.mul_ids[t], r + e);
                }
                const size_t at = (size_t)t * p.ldy + r;
                if (vec) {
                    if (EPI != EPI_GATED && EPI != EPI_GELU_MUL && p.resid) {
                        const float4 z = *reinterpret_cast<const float4 *>(p.resid + at);
                        o[0] += z.x; o[1] += z.y; o[2] += z.z; o[3] += z.w;
                    }
                    if (p.y_bf16) *reinterpret_cast<uint2 *>(static_cast<__nv_bfloat16 *>(p.y) + at) = make_uint2(bf16_pack(o[0], o[1]), bf16_pack(o[2], o[3]));
                    else *reinterpret_cast<float4 *>(static_cast<float *>(p.y) + at) = make_float4(o[0], o[1], o[2], o[3]);
                } else {
                    for (int e = 0; e < 4 && r + e < out_rows; ++e) {
                        if (EPI != EPI_GATED && EPI != EPI_GELU_MUL && p.resid) o[e] += p.resid[at + e];
                        if (p.y_bf16) static_cast<__nv_bfloat16 *>(p.y)[at + e] = __float2bfloat16_rn(o[e]);
                        else static_cast<float *>(p.y)[at + e] = o[e];
                    }
                }
            }
        }
        __syncwarp();
    }
}

template <int BN>
__global__ void __launch_bounds__(256, 1) linear_tc_kernel(const __grid_constant__ TcParams tp) {
    constexpr uint32_t NS = TcShape<BN>::NS, STAGE = TcShape<BN>::STAGE;
    extern __shared__ __align__(1024) uint8_t smem_raw[];
    uint8_t *smem = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    __shared__ uint64_t full[NS], empty[NS], acc_full[2], acc_empty[2];
    __shared__ uint32_t tmem_base_s, abort_s;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (tid == 0) {
        for (uint32_t s = 0; s < NS; ++s) {
            mbar_init(&full[s], 1);
            mbar_init(&empty[s], 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(&acc_full[i], 1);
            mbar_init(&acc_empty[i], 4);
        }
        abort_s = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 2) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base_s)), "r"(2u * BN) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    pdl_wait();
    pdl_launch();
    const uint32_t tmem = tmem_base_s;
    volatile uint32_t *abort_flag = &abort_s;
    auto wait = [&](uint64_t *bar, uint32_t parity) -> bool {
        for (uint32_t it = 0; it < TC_WAIT; ++it) {
            if (tc_mbar_try(bar, parity)) return true;
            if (*abort_flag) return false;
        }
        atomicExch(tp.status, 6u);
        *abort_flag = 1;
        return false;
    };
    auto locate = [&](uint32_t tile, uint32_t &row0, uint32_t &tok0) {
        uint32_t pi = 0;
        while (pi + 1 < tp.n && tile >= tp.tile_end[pi]) ++pi;
        const uint32_t k = tile - (pi ? tp.tile_end[pi - 1] : 0u);
        tok0 = k % tp.p[pi].tok_tiles * BM;
        row0 = k / tp.p[pi].tok_tiles * BN;
        return pi;
    };

    if (warp == 0) {
        if (lane == 0) {
            uint32_t k = 0;  // stages issued so far
            bool ok = true;
            for (uint32_t tile = blockIdx.x; tile < tp.tiles && ok; tile += gridDim.x) {
                uint32_t row0, tok0;
                const uint32_t pi = locate(tile, row0, tok0), ns0 = tp.p[pi].stages0, ns = tp.p[pi].stages;
                for (uint32_t j = 0; j < ns; ++j, ++k) {
                    const uint32_t s = k % NS;
                    if (k >= NS && !wait(&empty[s], ((k / NS) - 1) & 1)) {
                        ok = false;
                        break;
                    }
                    uint8_t *dst = smem + s * STAGE;
                    const uint32_t g = j >= ns0, c = (g ? j - ns0 : j) * BK;
                    mbar_expect_tx(&full[s], STAGE);
                    tma_load_2d(dst, &tp.x[pi][g], (int)c, (int)tok0, &full[s]);
                    tma_load_2d(dst + BM * BK * 2, &tp.w[pi][g], (int)c, (int)row0, &full[s]);
                }
            }
            if (*abort_flag)  // leaving early: let the copies in flight land first
                for (uint32_t i = k > NS ? k - NS : 0; i < k; ++i)
                    for (uint32_t it = 0; it < TC_WAIT && !tc_mbar_try(&full[i % NS], (i / NS) & 1); ++it) {}
        }
    } else if (warp == 1) {
        uint32_t k = 0, seq = 0;
        bool ok = true;
        for (uint32_t tile = blockIdx.x; tile < tp.tiles && ok; tile += gridDim.x, ++seq) {
            uint32_t row0, tok0;
            const uint32_t pi = locate(tile, row0, tok0), ns = tp.p[pi].stages, buf = seq & 1;
            if (seq >= 2) ok = wait(&acc_empty[buf], ((seq >> 1) - 1) & 1);
            ok = __all_sync(0xffffffffu, ok);
            for (uint32_t j = 0; j < ns && ok; ++j, ++k) {
                const uint32_t s = k % NS;
                ok = __all_sync(0xffffffffu, wait(&full[s], (k / NS) & 1));
                if (!ok) break;
                if (tc_elect_one()) {
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    const uint32_t a0 = smem_u32(smem + s * STAGE), b0 = a0 + BM * BK * 2;
#pragma unroll
                    for (uint32_t ks = 0; ks < BK / 16; ++ks)
                        tc_mma(tmem + buf * BN, tc_desc_kmajor(a0 + ks * 32), tc_desc_kmajor(b0 + ks * 32), tc_idesc_bf16(BM, BN), (j > 0 || ks > 0) ? 1u : 0u);
                    tc_commit(&empty[s]);
                    if (j + 1 == ns) tc_commit(&acc_full[buf]);
                }
                __syncwarp();
            }
        }
    } else if (warp >= 4) {
        const uint32_t q = warp & 3;
        float *stage = reinterpret_cast<float *>(smem + NS * STAGE) + q * 32 * EPI_LD;
        uint32_t seq = 0;
        bool ok = true;
        for (uint32_t tile = blockIdx.x; tile < tp.tiles && ok; tile += gridDim.x, ++seq) {
            uint32_t row0, tok0;
            const uint32_t pi = locate(tile, row0, tok0), buf = seq & 1;
            const TcProblem &p = tp.p[pi];
            ok = __all_sync(0xffffffffu, wait(&acc_full[buf], (seq >> 1) & 1));
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t ncol = min((uint32_t)BN, p.rows - row0), acc = tmem + buf * BN + ((q * 32u) << 16);
            if (tok0 + 32 * q < p.tokens) {
                const bool bare = !p.bias && !p.resid && p.scale == 1.0f && p.cap == 0.0f;
                if (p.act == LINEAR_ACT_GELU_TANH && p.mul && bare) tile_out<EPI_GELU_MUL>(p, acc, stage, row0, ncol, tok0 + 32 * q, lane);
                else if (p.act == LINEAR_ACT_SWIGLU) tile_out<EPI_GATED>(p, acc, stage, row0, ncol, tok0 + 32 * q, lane);
                else if (p.act == LINEAR_ACT_GELU_TANH || p.cap > 0.0f || p.mul) tile_out<EPI_ANY>(p, acc, stage, row0, ncol, tok0 + 32 * q, lane);
                else tile_out<EPI_PLAIN>(p, acc, stage, row0, ncol, tok0 + 32 * q, lane);
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) tc_mbar_arrive(&acc_empty[buf]);
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 2) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(2u * BN) : "memory");
    }
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *,
                                  const cuuint32_t *, const cuuint32_t *, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion,
                                  CUtensorMapFloatOOBfill);

template <int BN>
int32_t launch_tc(brasa_cmd *cmd, const LinearProblem *p, uint32_t n) {
    brasa_ctx *ctx = cmd->ctx;
    TcParams tp;
    memset(&tp, 0, sizeof tp);
    uint32_t tiles = 0;
    for (uint32_t i = 0; i < n; ++i) {
        const LinearProblem &q = p[i];
        TcProblem &d = tp.p[i];
        d.rows = q.rows;
        d.tokens = q.tokens;
        d.tok_tiles = (q.tokens + BM - 1) / BM;
        d.stages0 = (q.seg[0].cols + BK - 1) / BK;
        d.stages = d.stages0 + (q.seg[1].cols + BK - 1) / BK;
        d.y = q.y;
        d.ldy = q.ldy;
        d.y_bf16 = q.y_bf16;
        d.bias = q.bias;
        d.resid = q.resid;
        d.act = q.act;
        d.scale = q.scale;
        d.cap = q.cap;
        d.mul = q.mul;
        d.mul_ids = q.mul_ids;
        d.ldm = q.ldm;
        for (int s = 0; s < 2; ++s) {
            const LinearSeg &g = q.seg[s].cols ? q.seg[s] : q.seg[0];
            const uint64_t xd[2] = {g.cols, q.tokens}, xst[1] = {(uint64_t)g.ldx * 2}, wd[2] = {g.cols, q.rows}, wst[1] = {(uint64_t)g.ldw * 2};
            const uint32_t xb[2] = {BK, BM}, wb[2] = {BK, (uint32_t)BN};
            BRASA_TRY(brasa_tmap_bf16(ctx, &tp.x[i][s], 2, g.x, xd, xst, xb));
            BRASA_TRY(brasa_tmap_bf16(ctx, &tp.w[i][s], 2, g.w, wd, wst, wb));
        }
        tiles += d.tok_tiles * ((q.rows + BN - 1) / BN);
        tp.tile_end[i] = tiles;
    }
    tp.n = n;
    tp.tiles = tiles;
    tp.status = ctx->status;
    const size_t smem = TcShape<BN>::SMEM;
    BRASA_TRY(brasa_smem_optin(ctx, (const void *)linear_tc_kernel<BN>, smem));
    BRASA_CUDA(ctx, brasa_launch_dependent(ctx, linear_tc_kernel<BN>, dim3(std::min<uint32_t>(tiles, ctx->sm_count)), dim3(256), smem, tp));
    return brasa_post_launch(cmd, "linear_tc");
}

}  // namespace

int32_t brasa_tmap_bf16(brasa_ctx *ctx, CUtensorMap *map, uint32_t rank, const void *base, const uint64_t *dims, const uint64_t *strides,
                        const uint32_t *box) {
    static EncodeTiledFn fn = [] {
        void *f = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &f, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess) f = nullptr;
        return (EncodeTiledFn)f;
    }();
    if (!fn) return brasa_fail(ctx, BRASA_ECUDA, "cuTensorMapEncodeTiled is not available");
    cuuint64_t d[3], st[2];
    cuuint32_t b[3], es[3] = {1, 1, 1};
    for (uint32_t i = 0; i < rank; ++i) {
        d[i] = dims[i];
        b[i] = box[i];
        if (i + 1 < rank) st[i] = strides[i];
    }
    const CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, rank, const_cast<void *>(base), d, st, b, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                          CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return brasa_fail(ctx, BRASA_ECUDA, "cuTensorMapEncodeTiled failed (%d)", (int)r);
    return BRASA_OK;
}

int32_t brasa_linear_launch(brasa_cmd *cmd, const LinearProblem *ps, uint32_t count, bool x_f32) {
    brasa_ctx *ctx = cmd->ctx;
    LinearProblem p[LINEAR_MAX];
    uint32_t n = 0;
    BRASA_REQUIRE(ctx, count <= LINEAR_MAX, "linear: at most %u products in a group", LINEAR_MAX);
    for (uint32_t i = 0; i < count; ++i) {
        const LinearProblem &q = ps[i];
        if (q.tokens == 0 || q.rows == 0) continue;
        BRASA_REQUIRE(ctx, q.seg[0].cols > 0 && q.y && q.seg[0].x && q.seg[0].w && q.ldy >= q.out_rows(), "linear: empty or short product");
        BRASA_REQUIRE(ctx, q.act != LINEAR_ACT_SWIGLU || (q.rows % 64 == 0 && !q.bias && q.scale == 1.0f && q.cap == 0.0f), "linear: gated rows come in pairs of 32, without bias, scale and cap");
        BRASA_REQUIRE(ctx, q.act != LINEAR_ACT_SWIGLU || (!q.mul && !q.resid), "linear: gated rows take neither a factor nor a residual");
        BRASA_REQUIRE(ctx, !q.mul || q.mul_ids, "linear: a factor's rows need token ids");
        for (int s = 0; s < 2; ++s) {
            const LinearSeg &g = q.seg[s];
            if (!g.cols) continue;
            BRASA_REQUIRE(ctx, g.ldw >= g.cols && g.ldx >= g.cols && g.ldw % 8 == 0 && g.ldx % 8 == 0, "linear: leading dimensions must be multiples of 8");
            BRASA_REQUIRE(ctx, ((uintptr_t)g.x & 15) == 0 && ((uintptr_t)g.w & 15) == 0, "linear: misaligned operand");
        }
        BRASA_REQUIRE(ctx, ((uintptr_t)q.y & 15) == 0 && ((uintptr_t)q.resid & 15) == 0, "linear: misaligned output");
        p[n++] = q;
    }
    if (n == 0) return BRASA_OK;
    if (x_f32) {
        SimtParams sp;
        uint32_t tiles = 0;
        for (uint32_t i = 0; i < n; ++i) {
            sp.p[i] = p[i];
            tiles += (p[i].rows + TN - 1) / TN * ((p[i].tokens + TM - 1) / TM);
            sp.tile_end[i] = tiles;
        }
        sp.n = n;
        linear_f32_kernel<<<tiles, 256, 0, ctx->stream>>>(sp);
        return brasa_post_launch(cmd, "linear_f32");
    }
    // the widest tile that still gives every SM work
    auto tiles_of = [&](uint32_t bn) {
        uint32_t t = 0;
        for (uint32_t i = 0; i < n; ++i) t += (p[i].rows + bn - 1) / bn * ((p[i].tokens + BM - 1) / BM);
        return t;
    };
    if (tiles_of(256) >= (uint32_t)ctx->sm_count) return launch_tc<256>(cmd, p, n);
    if (tiles_of(128) >= (uint32_t)ctx->sm_count) return launch_tc<128>(cmd, p, n);
    return launch_tc<64>(cmd, p, n);
}

int32_t brasa_linear_gemv_launch(brasa_cmd *cmd, const GemvInput &in, const GemvProblem *ps, uint32_t n) {
    brasa_ctx *ctx = cmd->ctx;
    BRASA_REQUIRE(ctx, n >= 1 && n <= LINEAR_MAX, "gemv: 1 to %u products in a group", LINEAR_MAX);
    GemvDevParams g;
    memset(&g, 0, sizeof g);
    auto up8 = [](uint32_t v) { return (v + 7) / 8 * 8; };
    BRASA_REQUIRE(ctx, !in.y || (in.x && in.wy && in.x_out != in.x && in.norm != GEMV_LAYER_NORM), "gemv: a pending sum needs its weights, a place of its own and no layer norm");
    g.x = in.x;
    g.y = in.y;
    g.wy = in.wy;
    g.x_out = in.x_out;
    g.norm = in.norm;
    g.gated = in.gated;
    g.width = in.width;
    g.eps = in.eps;
    uint32_t off = 0;
    for (int i = 0; i < 2; ++i) {
        const bool used = in.x ? in.w[i] != nullptr || (in.norm == GEMV_PLAIN && i == 0) : in.v[i] != nullptr;
        if (!used) continue;
        BRASA_REQUIRE(ctx, !in.parts[i] || in.x || (in.vw[i] && in.len[i] % in.parts[i] == 0), "gemv: an input that does not divide into its parts");
        g.parts[i] = in.x ? 0u : in.parts[i];
        g.vw[i] = in.vw[i];
        g.vscale[i] = in.vscale[i];
        g.w[i] = in.w[i];
        g.b[i] = in.b[i];
        g.v[i] = in.v[i];
        g.len[i] = in.x ? in.width : in.len[i];
        g.off[i] = off;
        off += up8(g.len[i]);
        g.nin = i + 1;
    }
    g.x_floats = off;
    BRASA_REQUIRE(ctx, g.nin >= 1 && (g.nin == 1 || g.len[0] > 0) && (g.nin == 1 || !in.x || in.norm == GEMV_LAYER_NORM), "gemv: no input, or two forms of an RMS norm");
    uint32_t rows = 0;
    for (uint32_t i = 0; i < n; ++i) {
        const LinearProblem &q = ps[i].p;
        GemvDevProblem &d = g.p[i];
        for (int s = 0; s < 2; ++s) {
            const LinearSeg &sg = q.seg[s];
            if (!sg.cols) continue;
            const uint32_t k = ps[i].input[s];
            BRASA_REQUIRE(ctx, k < g.nin && sg.cols == g.len[k] && sg.ldw % 8 == 0 && sg.ldw >= sg.cols && ((uintptr_t)sg.w & 15) == 0, "gemv: product %u does not fit its input", i);
            d.w[s] = sg.w;
            d.ldw[s] = sg.ldw;
            d.cols8[s] = up8(sg.cols);
            d.xoff[s] = g.off[k];
        }
        if (!d.w[1]) d.w[1] = d.w[0];
        d.rows = q.rows;
        d.y = (float *)q.y;
        d.bias = q.bias;
        d.resid = q.resid;
        d.act = q.act;
        d.scale = q.scale;
        d.cap = q.cap;
        d.mul = q.mul;
        d.mul_id = q.mul_ids;
        d.ldm = q.ldm;
        BRASA_REQUIRE(ctx, q.act != LINEAR_ACT_SWIGLU && (!q.mul || q.mul_ids), "gemv: gated rows are formed by the next product; a factor needs the token's id");
        rows += q.rows;
        g.row_end[i] = rows;
    }
    g.n = n;
    g.total_rows = rows;
    const size_t smem = (size_t)g.x_floats * 4;
    BRASA_REQUIRE(ctx, rows > 0 && smem + 4096 <= ctx->smem_optin, "gemv: input of %u values is too long", g.x_floats);
    // how many warps share a row: what leaves the busiest warp the fewest batches
    uint32_t best = 1, best_cost = UINT32_MAX;
    for (uint32_t s = 1; s <= 8; s *= 2) {
        const uint32_t teams = (uint32_t)ctx->sm_count * GV_WARPS / s, step = GV_UNROLL * 256 * s;
        uint64_t batches = 0;
        for (uint32_t i = 0; i < n; ++i) batches += (uint64_t)g.p[i].rows * ((g.p[i].cols8[0] + step - 1) / step + (g.p[i].cols8[1] + step - 1) / step);
        const uint32_t rounds = (rows + teams - 1) / teams, cost = (uint32_t)(rounds * ((batches + rows - 1) / rows) * 16 + rounds * (s > 1 ? 4 : 1));
        if (cost < best_cost) {
            best_cost = cost;
            best = s;
        }
    }
    const uint32_t grid = std::min<uint32_t>((uint32_t)ctx->sm_count, (rows * best + GV_WARPS - 1) / GV_WARPS);
    const int form = !in.x ? IN_VECTORS : (in.norm == GEMV_LAYER_NORM ? IN_LAYER_NORM : IN_STREAM);
    auto launch = [&](void (*kernel)(GemvDevParams)) -> int32_t {
        BRASA_TRY(brasa_smem_optin(ctx, (const void *)kernel, std::max<size_t>(smem, 48 * 1024)));
        BRASA_CUDA(ctx, brasa_launch_dependent(ctx, kernel, dim3(grid), dim3(32 * GV_WARPS), smem, g));
        return BRASA_OK;
    };
#define GEMV_KERNELS(S) {linear_gemv_kernel<S, IN_VECTORS>, linear_gemv_kernel<S, IN_STREAM>, linear_gemv_kernel<S, IN_LAYER_NORM>}
    static void (*const kernels[4][3])(GemvDevParams) = {GEMV_KERNELS(1), GEMV_KERNELS(2), GEMV_KERNELS(4), GEMV_KERNELS(8)};
#undef GEMV_KERNELS
    BRASA_TRY(launch(kernels[best == 1 ? 0 : (best == 2 ? 1 : (best == 4 ? 2 : 3))][form]));
    return brasa_post_launch(cmd, "linear_gemv");
}

extern "C" int32_t brasa_k_linear(brasa_cmd *cmd, const brasa_linear *ps, uint32_t count, int32_t f32_inputs) {
    if (!cmd || !ps) return BRASA_EINVAL;
    brasa_ctx *ctx = cmd->ctx;
    BRASA_REQUIRE(ctx, count >= 1 && count <= LINEAR_MAX, "linear: 1 to %u products", LINEAR_MAX);
    LinearProblem q[LINEAR_MAX];
    const uint64_t xe = f32_inputs ? 4 : 2;
    for (uint32_t i = 0; i < count; ++i) {
        const brasa_linear &p = ps[i];
        BRASA_REQUIRE(ctx, p.rows > 0 && p.tokens > 0 && p.cols > 0 && p.ldy >= (p.act == BRASA_ACT_SWIGLU ? p.rows / 2 : p.rows), "linear: empty product");
        BRASA_REQUIRE(ctx, p.act >= BRASA_ACT_NONE && p.act <= BRASA_ACT_SWIGLU && p.cap >= 0.0f, "linear: unknown activation or negative cap");
        BRASA_REQUIRE(ctx, !p.mul.buf || (arg_fits(p.mul_ids, (uint64_t)p.tokens * 4) && p.ldm >= (p.act == BRASA_ACT_SWIGLU ? p.rows / 2 : p.rows) &&
                                          arg_fits(p.mul, (uint64_t)p.mul_rows * p.ldm * 2)),
                      "linear: mul or its ids too small");
        BRASA_REQUIRE(ctx, arg_fits(p.w, (uint64_t)p.rows * p.ldw * 2) && arg_fits(p.x, (uint64_t)p.tokens * p.ldx * xe), "linear: w or x too small");
        BRASA_REQUIRE(ctx, !p.cols2 || (arg_fits(p.w2, (uint64_t)p.rows * p.ldw2 * 2) && arg_fits(p.x2, (uint64_t)p.tokens * p.ldx2 * xe)), "linear: w2 or x2 too small");
        BRASA_REQUIRE(ctx, arg_fits(p.y, (uint64_t)p.tokens * p.ldy * (p.y_bf16 ? 2 : 4)), "linear: y too small");
        BRASA_REQUIRE(ctx, (!p.bias.buf || arg_fits(p.bias, (uint64_t)p.rows * 4)) && (!p.resid.buf || arg_fits(p.resid, (uint64_t)p.tokens * p.ldy * 4)), "linear: bias or resid too small");
        q[i].seg[0] = LinearSeg{(const uint16_t *)arg_ptr(p.w), p.ldw, arg_ptr(p.x), p.ldx, p.cols};
        if (p.cols2) q[i].seg[1] = LinearSeg{(const uint16_t *)arg_ptr(p.w2), p.ldw2, arg_ptr(p.x2), p.ldx2, p.cols2};
        q[i].rows = p.rows;
        q[i].tokens = p.tokens;
        q[i].y = arg_ptr(p.y);
        q[i].ldy = p.ldy;
        q[i].y_bf16 = p.y_bf16 != 0;
        q[i].bias = (const float *)arg_ptr(p.bias);
        q[i].resid = (const float *)arg_ptr(p.resid);
        q[i].act = p.act;
        q[i].scale = p.scale;
        q[i].cap = p.cap;
        q[i].mul = (const uint16_t *)arg_ptr(p.mul);
        q[i].ldm = p.ldm;
        q[i].mul_ids = (const uint32_t *)arg_ptr(p.mul_ids);
    }
    return brasa_linear_launch(cmd, q, count, f32_inputs != 0);
}
