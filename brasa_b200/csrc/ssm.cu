// State-space mixer with one decay per head (Mamba-2): the right side of "parallel". One projection gives [z | x | B | C | dt]; x, B
// and C pass a short causal convolution with bias and silu. A head keeps S [state][vdim]; with dt > 0 out of a softplus and the
// decay a = exp(-exp(A_log) dt), a token does
//   S <- a S + dt B x^T,  y = S^T C + D x
// and the output is y silu(z) in equal parts over their root mean squares, times a weight. B and C are shared by a group of heads.
//
// Many tokens, bf16 mode: chunks of 64. With L_t the running sum of log a inside the chunk and S the state before it,
//   y_t = exp(L_t) S^T C_t + sum_{s <= t} exp(L_t - L_s) dt_s (C_t . B_s) x_s + D x_t
//   S_next = exp(L_end) S + sum_s B_s (exp(L_end - L_s) dt_s x_s)^T
// ssm_conv_kernel: convolutions, dt, L. ssm_state_kernel: the second line through the chunks, one block per head and 16 value
// columns, the state in the accumulators; the state before every chunk goes out as two bf16 terms (16 bits and more).
// ssm_chunk_kernel: the first line, all chunks and heads side by side. Products on mma.sync with f32 accumulation; x, B and C are
// bf16, every f32 factor (states, weighted inputs, decayed scores) enters as two bf16 terms. ssm_out_kernel: the norm.
// 32-bit mode, and sizes beyond the products': ssm_scan_kernel, token by token in f32 FMA, then the same norm.
// One token: ssm_step_kernel; its output is normed by the product behind it (GemvInput::parts).
//
// Per-sequence state: S and the convolution's inputs as a ring (conv_device.cuh). Position 0 starts over by ignoring both.
#include <cuda_bf16.h>

#include "conv_device.cuh"
#include "stack.h"
#include "tc_device.cuh"

using namespace brasa_dev;

namespace {

struct SsmShape {
    uint32_t heads, groups, vdim, state, taps;
    uint32_t inner;         // heads * vdim
    uint32_t channels;      // of the convolution: inner + 2 groups * state
    uint32_t vp, np, ldx;   // vdim and state rounded up to 16; a row of x | B | C with every head and group padded to those
};

constexpr uint32_t SL = 64;  // tokens of a chunk

// padded column of x | B | C -> the convolution's channel, or UINT32_MAX in the padding
__device__ __forceinline__ uint32_t channel_of(const SsmShape &s, uint32_t pc) {
    if (pc < s.heads * s.vp) {
        const uint32_t h = pc / s.vp, e = pc - h * s.vp;
        return e < s.vdim ? h * s.vdim + e : UINT32_MAX;
    }
    pc -= s.heads * s.vp;
    const uint32_t g = pc / s.np, e = pc - g * s.np;
    return e < s.state ? s.inner + g * s.state + e : UINT32_MAX;
}

struct SsmConv {
    SsmShape s;
    ConvView cv;
    const float *x, *dt_raw;  // projections [tokens][ld]
    uint32_t ldc, lddt, tokens;
    const float *w, *bias, *dt_bias, *a_log;
    void *xbc;        // [tokens][ldx]
    float *dt, *run;  // [chunks][heads][SL]: dt and L; null: not wanted
};

// Block (16 tokens, 256 padded columns); the last blockIdx.y: dt and L of a chunk, a warp per head.
template <typename T>
__global__ void __launch_bounds__(256) ssm_conv_kernel(SsmConv p) {
    const SsmShape s = p.s;
    pdl_wait();
    pdl_launch();
    const uint32_t t0 = blockIdx.x * CONV_RUN, n = min(CONV_RUN, p.tokens - t0);
    if (blockIdx.y * 256 < s.ldx) {
        const uint32_t pc = blockIdx.y * 256 + threadIdx.x;
        if (pc >= s.ldx) return;
        const uint32_t c = channel_of(s, pc);
        T *out = (T *)p.xbc + (size_t)t0 * s.ldx + pc;
        if (c == UINT32_MAX) {
            for (uint32_t t = 0; t < n; ++t) elem_store(out + (size_t)t * s.ldx, 0.0f);
        } else {
            conv_chunk<sizeof(T) == 2>(p.x, p.ldc, c, p.w, p.bias[c], t0, n, p.cv, c, [&](uint32_t t, float v) { elem_store(out + (size_t)t * s.ldx, v); });
        }
        return;
    }
    if (t0 % SL) return;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (uint32_t h = warp; h < s.heads; h += 8) {
        const float a = -expf(p.a_log[h]);
        float dt[2], l[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const uint32_t t = t0 + lane + 32 * i;
            dt[i] = t < p.tokens ? softplus_f(p.dt_raw[(size_t)t * p.lddt + h] + p.dt_bias[h]) : 0.0f;
            l[i] = a * dt[i];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float up = __shfl_up_sync(0xffffffffu, l[i], o);
                if ((int)lane >= o) l[i] += up;
            }
        }
        l[1] += __shfl_sync(0xffffffffu, l[0], 31);
        const size_t at = ((size_t)(t0 / SL) * s.heads + h) * SL + lane;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            p.dt[at + 32 * i] = dt[i];
            p.run[at + 32 * i] = l[i];
        }
    }
}

// The run's last inputs of the convolution into the ring (the kernel that read the older ones has finished).
__device__ __forceinline__ void store_ring(const SsmShape &s, const float *x, uint32_t ldc, float *ring, uint32_t tokens, uint32_t pos0) {
    const uint32_t n = min(tokens, s.taps), step = gridDim.x * gridDim.y * blockDim.x;
    for (uint32_t ch = (blockIdx.y * gridDim.x + blockIdx.x) * blockDim.x + threadIdx.x; ch < s.channels; ch += step)
        for (uint32_t t = tokens - n; t < tokens; ++t) ring[(size_t)((pos0 + t) % s.taps) * s.channels + ch] = x[(size_t)t * ldc + ch];
}

// ---- products --------------------------------------------------------------------------------------------------------------
__device__ __forceinline__ void ldm4(uint32_t r[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldm4t(uint32_t r[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma_bf16(float c[4], const uint32_t a[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// x = hi + lo up to 2^-17 of x, two neighbours at a time
__device__ __forceinline__ void split2(float x0, float x1, uint32_t &hi, uint32_t &lo) {
    hi = bf16_pack(x0, x1);
    lo = bf16_pack(x0 - bf16_lo(hi), x1 - bf16_hi(hi));
}

typedef __nv_bfloat16 bf16;

// 16-byte pieces of rows of `per` of them, dealt out to a block's threads one behind the other
template <uint32_t THREADS>
struct Pieces {
    uint32_t row, at, per, drow, dat;
    __device__ __forceinline__ Pieces(uint32_t tid, uint32_t per_row) : row(tid / per_row), at(tid % per_row), per(per_row), drow(THREADS / per_row), dat(THREADS % per_row) {}
    __device__ __forceinline__ void next() {
        row += drow;
        at += dat;
        if (at >= per) {
            at -= per;
            ++row;
        }
    }
};
// tokens 0 .. n - 1 of a chunk from src (leading dimension ld) to dst (leading dimension ldd), zeros up to SL
template <uint32_t THREADS>
__device__ __forceinline__ void copy_tokens(Pieces<THREADS> p, bf16 *dst, uint32_t ldd, const bf16 *src, uint32_t ld, uint32_t n) {
    for (; p.row < SL; p.next()) {
        bf16 *d = dst + p.row * ldd + p.at * 8;
        if (p.row < n) cp16(d, src + (size_t)p.row * ld + p.at * 8);
        else *reinterpret_cast<uint4 *>(d) = make_uint4(0, 0, 0, 0);
    }
}

struct SsmState {
    SsmShape s;
    const bf16 *xbc;
    const float *dt, *run;
    const float *x;  // the convolution's inputs, for the ring
    uint32_t ldc;
    float *ring, *state;  // state [heads][state][vdim]
    bf16 *before;         // [chunks][heads][hi, lo][np][vp]
    uint32_t tokens, pos0;
};

constexpr uint32_t CB = 16, NB = 3;  // value columns of a block, chunks on their way

// TPW: 16 x 16 tiles of the state per warp
template <int TPW>
__global__ void __launch_bounds__(256) ssm_state_kernel(SsmState p) {
    extern __shared__ __align__(16) uint8_t sm_raw[];
    const SsmShape s = p.s;
    const uint32_t ldb = s.np + 8, h = blockIdx.x, g = h / (s.heads / s.groups), c0 = blockIdx.y * CB;
    constexpr uint32_t ldv = CB + 8;
    bf16 *bs = (bf16 *)sm_raw, *xs = bs + NB * SL * ldb, *xh = xs + NB * SL * ldv, *xl = xh + SL * ldv;
    float *lr = (float *)(xl + SL * ldv), *dts = lr + NB * SL;  // [NB][SL] each
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gr = lane >> 2, q = lane & 3;
    const uint32_t tiles = s.np / 16, chunks = (p.tokens + SL - 1) / SL;
    const Pieces<256> pb(tid, s.np / 8), px(tid, CB / 8);
    pdl_wait();
    pdl_launch();
    store_ring(s, p.x, p.ldc, p.ring, p.tokens, p.pos0);
    auto fetch = [&](uint32_t chunk) {  // (a group per chunk, empty past the end: the waits below count groups)
        if (chunk < chunks) {
            const uint32_t b = chunk % NB, t0 = chunk * SL, n = min(SL, p.tokens - t0);
            const bf16 *src = p.xbc + (size_t)t0 * s.ldx;
            copy_tokens(pb, bs + b * SL * ldb, ldb, src + s.heads * s.vp + g * s.np, s.ldx, n);
            copy_tokens(px, xs + b * SL * ldv, ldv, src + h * s.vp + c0, s.ldx, n);
            if (tid < 2 * SL) {
                const size_t at = ((size_t)chunk * s.heads + h) * SL + (tid & (SL - 1));
                cp4((tid < SL ? lr : dts) + b * SL + (tid & (SL - 1)), (tid < SL ? p.run : p.dt) + at);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0);
    fetch(1);
    // tile i of the warp: rows 16 (warp + 8 i) + gr and + 8 x columns 8 j + 2 q and + 1
    float acc[TPW][2][4];
    auto row_of = [&](int i, int e) { return 16 * (warp + 8 * i) + gr + 8 * (e >> 1); };
    auto col_of = [&](int j, int e) { return c0 + 8 * j + 2 * q + (e & 1); };
#pragma unroll
    for (int i = 0; i < TPW; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e)
                acc[i][j][e] = (p.pos0 != 0 && row_of(i, e) < s.state && col_of(j, e) < s.vdim) ? p.state[((size_t)h * s.state + row_of(i, e)) * s.vdim + col_of(j, e)] : 0.0f;
    for (uint32_t chunk = 0; chunk < chunks; ++chunk) {
        const uint32_t b = chunk % NB;
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();  // the chunk has arrived; everything of the chunk before has been read
        fetch(chunk + 2);
        const float end = lr[b * SL + SL - 1];
#pragma unroll
        for (uint32_t i = tid; i < SL * (CB / 2); i += 256) {
            const uint32_t t = i / (CB / 2), e = i % (CB / 2) * 2;
            const float w = __expf(end - lr[b * SL + t]) * dts[b * SL + t];
            const uint32_t x = *reinterpret_cast<const uint32_t *>(xs + (b * SL + t) * ldv + e);
            uint32_t hi, lo;
            split2(bf16_lo(x) * w, bf16_hi(x) * w, hi, lo);
            *reinterpret_cast<uint32_t *>(xh + t * ldv + e) = hi;
            *reinterpret_cast<uint32_t *>(xl + t * ldv + e) = lo;
        }
        const float fade = __expf(end);
        bf16 *out = p.before + ((size_t)chunk * s.heads + h) * 2 * s.np * s.vp;
#pragma unroll
        for (int i = 0; i < TPW; ++i)
            if (warp + 8 * i < tiles)
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    if (chunk > 0 || p.pos0 != 0)
#pragma unroll
                        for (int e = 0; e < 4; e += 2) {
                            uint32_t hi, lo;
                            split2(acc[i][j][e], acc[i][j][e + 1], hi, lo);
                            uint32_t *dst = reinterpret_cast<uint32_t *>(out + (size_t)row_of(i, e) * s.vp + col_of(j, e));
                            dst[0] = hi;
                            dst[s.np * s.vp / 2] = lo;
                        }
#pragma unroll
                    for (int e = 0; e < 4; ++e) acc[i][j][e] *= fade;
                }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < TPW; ++i) {
            const uint32_t n0 = 16 * (warp + 8 * i);
            if (n0 >= s.np) break;
#pragma unroll
            for (uint32_t k0 = 0; k0 < SL; k0 += 16) {
                uint32_t a[4], bh[4], bl[4];
                ldm4t(a, smem_u32(bs + (b * SL + k0 + (lane & 7) + (lane >> 4) * 8) * ldb + n0 + ((lane >> 3) & 1) * 8));
                const uint32_t at = (k0 + (lane & 7) + ((lane >> 3) & 1) * 8) * ldv + (lane >> 4) * 8;
                ldm4t(bh, smem_u32(xh + at));
                ldm4t(bl, smem_u32(xl + at));
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    mma_bf16(acc[i][j], a, bl[2 * j], bl[2 * j + 1]);
                    mma_bf16(acc[i][j], a, bh[2 * j], bh[2 * j + 1]);
                }
            }
        }
    }
#pragma unroll
    for (int i = 0; i < TPW; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (row_of(i, e) < s.state && col_of(j, e) < s.vdim) p.state[((size_t)h * s.state + row_of(i, e)) * s.vdim + col_of(j, e)] = acc[i][j][e];
}

struct SsmChunk {
    SsmShape s;
    const bf16 *xbc, *before;
    const float *dt, *run, *z, *D;
    uint32_t ldz;
    float *y;  // [tokens][inner], times silu(z)
    uint32_t tokens;
    bool empty;  // the state before the first chunk is zero
};

// Block: one chunk of one head, warps w and w + 4 = tokens 16 w .. 16 w + 15, each half of the value columns. VT: 16-wide blocks
// of a warp's columns, at most.
template <int VT>
__global__ void __launch_bounds__(256, 2) ssm_chunk_kernel(SsmChunk p) {
    extern __shared__ __align__(16) uint8_t sm_raw[];
    const SsmShape s = p.s;
    const uint32_t ldb = s.np + 8, ldv = s.vp + 8, chunk = blockIdx.x, h = blockIdx.y, g = h / (s.heads / s.groups), t0 = chunk * SL, n = min(SL, p.tokens - t0);
    bf16 *cs = (bf16 *)sm_raw, *bs = cs + SL * ldb, *xs = bs + SL * ldb, *sh = xs + SL * ldv, *sl = sh + s.np * ldv;
    float *lr = (float *)(sl + s.np * ldv), *dts = lr + SL;
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = (tid >> 5) & 3, gr = lane >> 2, q = lane & 3;
    const uint32_t vt = s.vp / 16, v0 = tid < 128 ? 0u : (vt + 1) / 2, nv = tid < 128 ? (vt + 1) / 2 : vt / 2;  // this warp's blocks of value columns
    const bool inter = chunk > 0 || !p.empty;
    pdl_wait();
    pdl_launch();
    {
        const bf16 *src = p.xbc + (size_t)t0 * s.ldx;
        const uint32_t bo = s.heads * s.vp + g * s.np;
        const Pieces<256> pn(tid, s.np / 8), pv(tid, s.vp / 8);
        copy_tokens(pn, cs, ldb, src + bo + s.groups * s.np, s.ldx, n);
        copy_tokens(pn, bs, ldb, src + bo, s.ldx, n);
        copy_tokens(pv, xs, ldv, src + h * s.vp, s.ldx, n);
        if (tid < 2 * SL) cp4((tid < SL ? lr : dts) + (tid & (SL - 1)), (tid < SL ? p.run : p.dt) + ((size_t)chunk * s.heads + h) * SL + (tid & (SL - 1)));
        if (inter) {
            const bf16 *st = p.before + ((size_t)chunk * s.heads + h) * 2 * s.np * s.vp;
            for (Pieces<256> r = pv; r.row < 2 * s.np; r.next()) cp16(sh + r.row * ldv + r.at * 8, st + (size_t)r.row * s.vp + r.at * 8);  // (lo rows follow the hi rows in both)
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    float y[VT][2][4] = {}, G[8][4] = {};
    const uint32_t row0 = 16 * warp;
    for (uint32_t k0 = 0; k0 < s.np; k0 += 16) {
        uint32_t a[4];
        ldm4(a, smem_u32(cs + (row0 + (lane & 7) + ((lane >> 3) & 1) * 8) * ldb + k0 + (lane >> 4) * 8));
#pragma unroll
        for (uint32_t j = 0; j < 4; ++j)
            if (j <= warp) {
                uint32_t b[4];
                ldm4(b, smem_u32(bs + (16 * j + (lane & 7) + (lane >> 4) * 8) * ldb + k0 + ((lane >> 3) & 1) * 8));
                mma_bf16(G[2 * j], a, b[0], b[1]);
                mma_bf16(G[2 * j + 1], a, b[2], b[3]);
            }
        if (inter)
#pragma unroll
            for (int c = 0; c < VT; ++c)
                if (c < (int)nv) {
                    const uint32_t at = (k0 + (lane & 7) + ((lane >> 3) & 1) * 8) * ldv + 16 * (v0 + c) + (lane >> 4) * 8;
                    uint32_t bh[4], bl[4];
                    ldm4t(bh, smem_u32(sh + at));
                    ldm4t(bl, smem_u32(sl + at));
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        mma_bf16(y[c][j], a, bl[2 * j], bl[2 * j + 1]);
                        mma_bf16(y[c][j], a, bh[2 * j], bh[2 * j + 1]);
                    }
                }
    }
    const float l0 = lr[row0 + gr], l1 = lr[row0 + gr + 8];
    if (inter) {
        const float f0 = __expf(l0), f1 = __expf(l1);
#pragma unroll
        for (int c = 0; c < VT; ++c)
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                y[c][j][0] *= f0;
                y[c][j][1] *= f0;
                y[c][j][2] *= f1;
                y[c][j][3] *= f1;
            }
    }
#pragma unroll
    for (uint32_t j = 0; j < 4; ++j)
        if (j <= warp) {
            uint32_t ah[4], al[4];
#pragma unroll
            for (int half = 0; half < 2; ++half) {  // eight tokens s of the sixteen
                const uint32_t c = 16 * j + 8 * half + 2 * q;
                const float *gg = G[2 * j + half];
                float m[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const uint32_t t = row0 + gr + 8 * (e >> 1), ss = c + (e & 1);
                    m[e] = ss <= t ? gg[e] * __expf((e >> 1 ? l1 : l0) - lr[ss]) * dts[ss] : 0.0f;
                }
                split2(m[0], m[1], ah[2 * half], al[2 * half]);
                split2(m[2], m[3], ah[2 * half + 1], al[2 * half + 1]);
            }
#pragma unroll
            for (int c = 0; c < VT; ++c)
                if (c < (int)nv) {
                    uint32_t b[4];
                    ldm4t(b, smem_u32(xs + (16 * j + (lane & 7) + ((lane >> 3) & 1) * 8) * ldv + 16 * (v0 + c) + (lane >> 4) * 8));
#pragma unroll
                    for (int k = 0; k < 2; ++k) {
                        mma_bf16(y[c][k], al, b[2 * k], b[2 * k + 1]);
                        mma_bf16(y[c][k], ah, b[2 * k], b[2 * k + 1]);
                    }
                }
        }
    const float D = p.D[h];
    const bool pair = (s.vdim & 1) == 0 && (p.ldz & 1) == 0;
#pragma unroll
    for (int c = 0; c < VT; ++c)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
                const uint32_t t = row0 + gr + 4 * e, col = 16 * (v0 + c) + 8 * j + 2 * q;
                if (c >= (int)nv || t >= n || col >= s.vdim) continue;
                const uint32_t x = *reinterpret_cast<const uint32_t *>(xs + t * ldv + col);
                const float v0 = fmaf(D, bf16_lo(x), y[c][j][e]), v1 = fmaf(D, bf16_hi(x), y[c][j][e + 1]);
                const float *z = p.z + (size_t)(t0 + t) * p.ldz + h * s.vdim + col;
                float *dst = p.y + (size_t)(t0 + t) * s.inner + h * s.vdim + col;
                if (pair) {
                    const float2 zz = *reinterpret_cast<const float2 *>(z);
                    *reinterpret_cast<float2 *>(dst) = make_float2(v0 * silu_fast(zz.x), v1 * silu_fast(zz.y));
                } else {
                    dst[0] = v0 * silu_fast(z[0]);
                    if (col + 1 < s.vdim) dst[1] = v1 * silu_fast(z[1]);
                }
            }
}

// ---- token by token in f32 ---------------------------------------------------------------------------------------------------
struct SsmScan {
    SsmShape s;
    const void *xbc;
    const float *x, *dt_raw, *dt_bias, *a_log, *z, *D;
    uint32_t ldc, lddt, ldz;
    float *ring, *state, *y;
    uint32_t tokens, pos0;
};
constexpr uint32_t ST = 32;  // tokens between two exchanges

// Block: 32 value columns (lanes) of one head; warp w keeps the state's rows w, w + 8, .. (R of them at most).
template <typename T, int R>
__global__ void __launch_bounds__(256) ssm_scan_kernel(SsmScan p) {
    extern __shared__ __align__(16) float sm[];
    const SsmShape s = p.s;
    float *bs = sm, *cs = bs + ST * s.np, *part = cs + ST * s.np, *xs = part + 8 * ST * 32, *as = xs + ST * 32, *dts = as + ST;
    const uint32_t h = blockIdx.x, g = h / (s.heads / s.groups), c0 = blockIdx.y * 32, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    pdl_wait();
    pdl_launch();
    store_ring(s, p.x, p.ldc, p.ring, p.tokens, p.pos0);
    const bool col = c0 + lane < s.vdim;
    float S[R];
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const uint32_t row = warp + 8 * i;
        S[i] = (p.pos0 != 0 && col && row < s.state) ? p.state[((size_t)h * s.state + row) * s.vdim + c0 + lane] : 0.0f;
    }
    const uint32_t bo = s.heads * s.vp + g * s.np, co = bo + s.groups * s.np, xo = h * s.vp + c0;
    const float a = -expf(p.a_log[h]);
    for (uint32_t t0 = 0; t0 < p.tokens; t0 += ST) {
        const uint32_t n = min(ST, p.tokens - t0);
        const T *src = (const T *)p.xbc + (size_t)t0 * s.ldx;
        for (uint32_t i = tid; i < n * s.np; i += 256) {
            const uint32_t t = i / s.np, e = i - t * s.np;
            bs[i] = elem_load(src + (size_t)t * s.ldx + bo + e);
            cs[i] = elem_load(src + (size_t)t * s.ldx + co + e);
        }
        for (uint32_t i = tid; i < n * 32; i += 256) xs[i] = c0 + (i & 31) < s.vdim ? elem_load(src + (size_t)(i >> 5) * s.ldx + xo + (i & 31)) : 0.0f;
        if (tid < n) {
            dts[tid] = softplus_f(p.dt_raw[(size_t)(t0 + tid) * p.lddt + h] + p.dt_bias[h]);
            as[tid] = expf(a * dts[tid]);
        }
        __syncthreads();
        for (uint32_t t = 0; t < n; ++t) {
            const float f = as[t], x = dts[t] * xs[t * 32 + lane];
            float y = 0.0f;
#pragma unroll
            for (int i = 0; i < R; ++i) {
                const uint32_t row = warp + 8 * i;
                if (row < s.state) {
                    S[i] = fmaf(bs[t * s.np + row], x, S[i] * f);
                    y = fmaf(S[i], cs[t * s.np + row], y);
                }
            }
            part[(warp * ST + t) * 32 + lane] = y;
        }
        __syncthreads();
        for (uint32_t i = tid; i < n * 32; i += 256) {
            const uint32_t t = i >> 5, e = i & 31;
            if (c0 + e >= s.vdim) continue;
            float y = p.D[h] * xs[i];
            for (uint32_t w = 0; w < 8; ++w) y += part[(w * ST + t) * 32 + e];
            p.y[(size_t)(t0 + t) * s.inner + h * s.vdim + c0 + e] = y * silu_f(p.z[(size_t)(t0 + t) * p.ldz + h * s.vdim + c0 + e]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const uint32_t row = warp + 8 * i;
        if (col && row < s.state) p.state[((size_t)h * s.state + row) * s.vdim + c0 + lane] = S[i];
    }
}

// y in equal parts over their root mean squares, times w and f. Block: one part of one token.
template <typename T>
__global__ void __launch_bounds__(256) ssm_out_kernel(const float *y, const float *w, T *out, uint32_t inner, uint32_t parts, uint32_t ldo, float eps, float f) {
    __shared__ float red[8];
    pdl_wait();
    pdl_launch();
    const uint32_t n = inner / parts, o = blockIdx.y * n, tid = threadIdx.x;
    const float *src = y + (size_t)blockIdx.x * inner + o;
    T *dst = out + (size_t)blockIdx.x * ldo + o;
    float ss = 0.0f;
    const bool vec = ((n | inner | ldo) & 3) == 0;
    if (vec) {
        for (uint32_t i = tid; i < n / 4; i += 256) {
            const float4 v = reinterpret_cast<const float4 *>(src)[i];
            ss += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
        }
    } else {
        for (uint32_t i = tid; i < n; i += 256) ss = fmaf(src[i], src[i], ss);
    }
    ss = warp_sum(ss);
    if ((tid & 31) == 0) red[tid >> 5] = ss;
    __syncthreads();
    ss = ((red[0] + red[1]) + (red[2] + red[3])) + ((red[4] + red[5]) + (red[6] + red[7]));
    const float inv = f / sqrtf(ss / (float)n + eps);
    if (vec) {
        for (uint32_t i = tid; i < n / 4; i += 256) {
            const float4 v = reinterpret_cast<const float4 *>(src)[i], k = reinterpret_cast<const float4 *>(w + o)[i];
            const float4 r = make_float4(v.x * inv * k.x, v.y * inv * k.y, v.z * inv * k.z, v.w * inv * k.w);
            if (sizeof(T) == 4) reinterpret_cast<float4 *>(dst)[i] = r;
            else reinterpret_cast<uint2 *>(dst)[i] = make_uint2(bf16_pack(r.x, r.y), bf16_pack(r.z, r.w));
        }
    } else {
        for (uint32_t i = tid; i < n; i += 256) elem_store(dst + i, src[i] * inv * w[o + i]);
    }
}

// ---- one token ---------------------------------------------------------------------------------------------------------------
struct SsmStep {
    SsmShape s;
    const float *x, *dt_raw, *z;  // projections of this token
    const float *w, *bias, *dt_bias, *a_log, *D;
    float *ring, *state, *y;      // y [inner], times silu(z)
    const uint32_t *pos;
};

constexpr uint32_t SW = 16;  // warps of a block

// Block: 32 value columns (lanes) of one head; warp w owns the state's rows w, w + SW, .., which are read ahead of the kernel
// before this one: the last to write them was the token before.
template <int R>
__global__ void __launch_bounds__(32 * SW) ssm_step_kernel(SsmStep p) {
    extern __shared__ __align__(16) float sm[];
    const SsmShape s = p.s;
    float *bs = sm, *cs = bs + s.state, *xs = cs + s.state, *part = xs + 32;
    const uint32_t h = blockIdx.x, share = s.heads / s.groups, g = h / share, c0 = blockIdx.y * 32, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const bool col = c0 + lane < s.vdim;
    float *state = p.state + (size_t)h * s.state * s.vdim + c0 + lane;
    float S[R];
#pragma unroll
    for (int i = 0; i < R; ++i) S[i] = (col && warp + SW * i < s.state) ? state[(size_t)(warp + SW * i) * s.vdim] : 0.0f;
    pdl_wait();
    pdl_launch();
    const uint32_t pos = *p.pos, slot = pos % s.taps, nx = min(32u, s.vdim - c0);
    const ConvView cv{p.ring, s.channels, s.taps, pos};
    const bool keeper = h % share == 0 && blockIdx.y == 0;  // stores the group's B and C inputs (nobody reads this row in this step)
    for (uint32_t i = tid; i < 2 * s.state + nx; i += 32 * SW) {
        const uint32_t c = i < s.state ? s.inner + g * s.state + i
                                       : (i < 2 * s.state ? s.inner + (s.groups + g) * s.state + i - s.state : h * s.vdim + c0 + i - 2 * s.state);
        (i < s.state ? bs[i] : (i < 2 * s.state ? cs[i - s.state] : xs[i - 2 * s.state])) = silu_f(conv_step(p.x, c, p.w, cv, slot, c) + p.bias[c]);
        if (keeper || i >= 2 * s.state) p.ring[(size_t)slot * s.channels + c] = p.x[c];
    }
    const float dt = softplus_f(p.dt_raw[h] + p.dt_bias[h]), f = pos == 0 ? 0.0f : expf(-expf(p.a_log[h]) * dt);
    __syncthreads();
    const float x = col ? dt * xs[lane] : 0.0f;
    float y = 0.0f;
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const uint32_t row = warp + SW * i;
        if (row < s.state) {
            S[i] = fmaf(bs[row], x, pos == 0 ? 0.0f : S[i] * f);
            y = fmaf(S[i], cs[row], y);
            if (col) state[(size_t)row * s.vdim] = S[i];
        }
    }
    part[warp * 32 + lane] = y;
    __syncthreads();
    if (tid < nx) {
        y = p.D[h] * xs[tid];
        for (uint32_t w = 0; w < SW; ++w) y += part[w * 32 + tid];
        p.y[h * s.vdim + c0 + tid] = y * silu_f(p.z[h * s.vdim + c0 + tid]);
    }
}

}  // namespace

namespace brasa_stack {
namespace {

class StateSpace : public Mixer {
  public:
    bool configure(const brasa::Json &c, uint32_t width, float eps, std::string &err) override {
        if (!read_u32(c, "heads", &s_.heads, err) || !read_u32(c, "vdim", &s_.vdim, err) || !read_u32(c, "state", &s_.state, err) ||
            !read_u32(c, "groups", &s_.groups, err) || !read_u32(c, "conv", &s_.taps, err) || !read_u32(c, "norm_groups", &parts_, err))
            return false;
        if (s_.heads % s_.groups) return err = "state space: heads must be a multiple of groups", false;
        s_.inner = s_.heads * s_.vdim;
        if (s_.inner % parts_) return err = "state space: norm_groups must divide heads * vdim", false;
        if (s_.state > 512 || s_.vdim > 1024) return err = "state space: state up to 512, vdim up to 1024", false;
        s_.channels = s_.inner + 2 * s_.groups * s_.state;
        s_.vp = (s_.vdim + 15) / 16 * 16;
        s_.np = (s_.state + 15) / 16 * 16;
        s_.ldx = s_.heads * s_.vp + 2 * s_.groups * s_.np;
        width_ = width;
        eps_ = eps;
        return true;
    }
    bool scale_output(float f) override {
        factor_ = f;
        return true;
    }

    int32_t build(Builder &b, const std::string &x) override {
        BRASA_TRY(b.matrix(x + "in", s_.inner + s_.channels + s_.heads, width_, &in_));
        outs.resize(1);
        BRASA_TRY(b.matrix(x + "o", width_, s_.inner, &outs[0]));
        BRASA_TRY(b.vector(x + "conv", (uint64_t)s_.channels * s_.taps, &w_));
        BRASA_TRY(b.vector(x + "conv.b", s_.channels, &bias_));
        BRASA_TRY(b.vector(x + "dt_bias", s_.heads, &dt_bias_));
        BRASA_TRY(b.vector(x + "A_log", s_.heads, &a_log_));
        BRASA_TRY(b.vector(x + "D", s_.heads, &d_));
        BRASA_TRY(b.vector(x + "norm", s_.inner, &norm_));
        outs[0].parts = parts_;
        outs[0].part_w = norm_;
        outs[0].part_scale = factor_;
        BRASA_TRY(b.get(Builder::STATE, 4ull * s_.taps * s_.channels, (void **)&ring_));
        BRASA_TRY(b.get(Builder::STATE, 4ull * s_.heads * s_.state * s_.vdim, (void **)&state_));
        const uint64_t t = b.limits.max_tokens, chunks = (t + SL - 1) / SL;
        ldz_ = up8(s_.inner);
        ldc_ = up8(s_.channels);
        lddt_ = up8(s_.heads);
        const bool products = !b.f32 && fits();
        Carver c;
        at_.z = c.take(4 * t * ldz_);
        at_.c = c.take(4 * t * ldc_);
        at_.dt_raw = c.take(4 * t * lddt_);
        at_.xbc = c.take(t * s_.ldx * b.elem());
        at_.y = c.take(4 * t * s_.inner);
        at_.dt = c.take(products ? 4 * chunks * s_.heads * SL : 0);
        at_.run = c.take(products ? 4 * chunks * s_.heads * SL : 0);
        at_.before = c.take(products ? 2 * chunks * s_.heads * 2 * s_.np * s_.vp : 0);
        at_.total = c.at;
        return BRASA_OK;
    }

    uint64_t scratch_bytes() const override { return at_.total; }

    void project(const Run &r, std::vector<GemvProblem> &out) override {
        auto rows = [&](uint32_t first, uint32_t n) {
            Weight w = in_;
            w.p += (size_t)first * in_.ld;
            w.rows = n;
            return w;
        };
        add_projection(r, rows(0, s_.inner), at_.z, ldz_, out);
        add_projection(r, rows(s_.inner, s_.channels), at_.c, ldc_, out);
        add_projection(r, rows(s_.inner + s_.channels, s_.heads), at_.dt_raw, lddt_, out);
    }

    int32_t mix(const Run &r) override {
        if (r.dev_pos) return step(r);
        return r.f32 ? run<float>(r) : run<bf16>(r);
    }

  private:
    bool fits() const { return s_.np <= 256 && s_.vp <= 128; }

    template <typename T>
    int32_t run(const Run &r) {
        brasa_ctx *ctx = r.cmd->ctx;
        auto f = [&](uint64_t at) { return (float *)(r.scratch + at); };
        const bool products = !r.f32 && fits();
        const uint32_t chunks = (r.tokens + SL - 1) / SL;
        SsmConv cp{s_, ConvView{ring_, s_.channels, s_.taps, r.pos0}, f(at_.c), f(at_.dt_raw), ldc_, lddt_, r.tokens, w_, bias_, dt_bias_, a_log_, r.scratch + at_.xbc,
                   f(at_.dt), f(at_.run)};
        BRASA_CUDA(ctx, brasa_launch_dependent(ctx, ssm_conv_kernel<T>, dim3((r.tokens + CONV_RUN - 1) / CONV_RUN, (s_.ldx + 255) / 256 + (products ? 1 : 0)), dim3(256), 0, cp));
        BRASA_TRY(brasa_post_launch(r.cmd, "ssm_conv"));
        if (products) {
            const bf16 *xbc = (const bf16 *)(r.scratch + at_.xbc);
            bf16 *before = (bf16 *)(r.scratch + at_.before);
            SsmState sp{s_, xbc, f(at_.dt), f(at_.run), f(at_.c), ldc_, ring_, state_, before, r.tokens, r.pos0};
            const size_t ssm = (size_t)(NB * SL * (s_.np + 8) + (NB + 2) * SL * (CB + 8)) * 2 + 2 * NB * SL * 4;
            const dim3 grid(s_.heads, s_.vp / CB);
            auto state = s_.np <= 128 ? ssm_state_kernel<1> : ssm_state_kernel<2>;
            BRASA_TRY(brasa_smem_optin(ctx, (const void *)state, std::max<size_t>(ssm, 48 * 1024)));
            BRASA_CUDA(ctx, brasa_launch_dependent(ctx, state, grid, dim3(256), ssm, sp));
            BRASA_TRY(brasa_post_launch(r.cmd, "ssm_state"));
            SsmChunk kp{s_, xbc, before, f(at_.dt), f(at_.run), f(at_.z), d_, ldz_, f(at_.y), r.tokens, r.pos0 == 0};
            const size_t csm = (size_t)(2 * SL * (s_.np + 8) + (SL + 2 * s_.np) * (s_.vp + 8)) * 2 + 2 * SL * 4;
            BRASA_REQUIRE(ctx, csm + 1024 <= ctx->smem_optin, "state space: sizes too large");
            auto chunk = s_.vp <= 64 ? ssm_chunk_kernel<2> : ssm_chunk_kernel<4>;
            BRASA_TRY(brasa_smem_optin(ctx, (const void *)chunk, std::max<size_t>(csm, 48 * 1024)));
            BRASA_CUDA(ctx, brasa_launch_dependent(ctx, chunk, dim3(chunks, s_.heads), dim3(256), csm, kp));
            BRASA_TRY(brasa_post_launch(r.cmd, "ssm_chunk"));
        } else {
            SsmScan sp{s_, r.scratch + at_.xbc, f(at_.c), f(at_.dt_raw), dt_bias_, a_log_, f(at_.z), d_, ldc_, lddt_, ldz_, ring_, state_, f(at_.y), r.tokens, r.pos0};
            const size_t smem = (size_t)(2 * ST * s_.np + 8 * ST * 32 + ST * 32 + 2 * ST) * 4;
            BRASA_REQUIRE(ctx, smem + 1024 <= ctx->smem_optin, "state space: sizes too large");
            auto scan = s_.state <= 128 ? ssm_scan_kernel<T, 16> : (s_.state <= 256 ? ssm_scan_kernel<T, 32> : ssm_scan_kernel<T, 64>);
            BRASA_TRY(brasa_smem_optin(ctx, (const void *)scan, std::max<size_t>(smem, 48 * 1024)));
            BRASA_CUDA(ctx, brasa_launch_dependent(ctx, scan, dim3(s_.heads, (s_.vdim + 31) / 32), dim3(256), smem, sp));
            BRASA_TRY(brasa_post_launch(r.cmd, "ssm_scan"));
        }
        BRASA_CUDA(ctx, brasa_launch_dependent(ctx, ssm_out_kernel<T>, dim3(r.tokens, parts_), dim3(256), 0, f(at_.y), norm_, (T *)r.out[0], s_.inner, parts_, r.ldo[0], eps_, factor_));
        return brasa_post_launch(r.cmd, "ssm_out");
    }

    int32_t step(const Run &r) {
        brasa_ctx *ctx = r.cmd->ctx;
        auto f = [&](uint64_t at) { return (float *)(r.scratch + at); };
        SsmStep p{s_, f(at_.c), f(at_.dt_raw), f(at_.z), w_, bias_, dt_bias_, a_log_, d_, ring_, state_, (float *)r.out[0], r.dev_pos};
        const size_t smem = (size_t)(2 * s_.state + 32 + SW * 32) * 4;
        auto kernel = s_.state <= 128 ? ssm_step_kernel<8> : (s_.state <= 256 ? ssm_step_kernel<16> : ssm_step_kernel<32>);
        BRASA_CUDA(ctx, brasa_launch_dependent(ctx, kernel, dim3(s_.heads, (s_.vdim + 31) / 32), dim3(32 * SW), smem, p));
        return brasa_post_launch(r.cmd, "ssm_step");
    }

    SsmShape s_{};
    uint32_t width_ = 0, parts_ = 1, ldz_ = 0, ldc_ = 0, lddt_ = 0;
    float eps_ = 0.0f, factor_ = 1.0f;
    Weight in_;
    const float *w_ = nullptr, *bias_ = nullptr, *dt_bias_ = nullptr, *a_log_ = nullptr, *d_ = nullptr, *norm_ = nullptr;
    float *ring_ = nullptr, *state_ = nullptr;
    struct {
        uint64_t z, c, dt_raw, xbc, y, dt, run, before, total;
    } at_{};
};

}  // namespace

std::unique_ptr<Mixer> make_state_space() { return std::unique_ptr<Mixer>(new StateSpace()); }

}  // namespace brasa_stack
