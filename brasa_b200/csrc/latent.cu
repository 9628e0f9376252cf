// Latent attention inside a sliding window ("latent_attention"): keys and values are linear maps of one normed latent vector per
// token, plus one rotated key part shared by all heads, so the cache holds kv_rank + rot_dim values per token and layer.
//
// Cache: a ring of rows, position p in row p % rows, rows >= window - 1 + the longest run: a run's own tokens never push out
// what its first query still sees.
// Many tokens: the latents of the visible positions are expanded to keys and values per head by two products, and
// window_attn.cu attends over them.
// One token: nothing is expanded. latent_absorb_kernel takes the query through the key map (q_lat = W_uk^T q),
// latent_partial_kernel attends over the latent rows themselves, split over blocks of keys, for eight heads per block, and
// latent_combine_kernel merges the parts and takes each head's latent sum through the value map.
#include <cuda_bf16.h>

#include "stack.h"
#include "tc_device.cuh"
#include "window_attn.h"

using namespace brasa_dev;

namespace {

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

struct LatentShape {
    uint32_t heads, dim, rot, rot_dims, vdim, kr, window;
    uint32_t rows, ldc, ldr;  // the ring: rows, leading dimensions of its two parts
    float scale, eps;
};

__device__ __forceinline__ float rot_elem(const float *x, uint32_t e, uint32_t dims, const float *c, const float *s) {
    const uint32_t half = dims / 2;
    if (e < half) return x[e] * c[e] - x[e + half] * s[e];
    if (e < dims) return x[e] * c[e - half] + x[e - half] * s[e - half];
    return x[e];
}

// One token's row of the ring from its down projection `d`: the latent divided by its root mean square, the shared key part
// rotated. A block of 256 threads.
template <typename T>
__device__ __forceinline__ void store_row(const LatentShape &s, const float *d, uint32_t pos, const float *w, const float *cos_t, const float *sin_t, T *c, T *r) {
    __shared__ float red[8];
    float ss = 0.0f;
    for (uint32_t i = threadIdx.x; i < s.kr; i += 256) ss = fmaf(d[i], d[i], ss);
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.0f;
    for (int i = 0; i < 8; ++i) ss += red[i];
    const float inv = 1.0f / sqrtf(ss / (float)s.kr + s.eps);
    const uint32_t slot = pos % s.rows, half = s.rot_dims / 2;
    for (uint32_t i = threadIdx.x; i < s.kr; i += 256) elem_store(c + (size_t)slot * s.ldc + i, d[i] * inv * w[i]);
    for (uint32_t i = threadIdx.x; i < s.rot; i += 256)
        elem_store(r + (size_t)slot * s.ldr + i, rot_elem(d + s.kr, i, s.rot_dims, cos_t + (size_t)pos * half, sin_t + (size_t)pos * half));
}

// Many tokens: one warp per token, its latent in registers (up to 1024 wide).
template <typename T>
__global__ void __launch_bounds__(256) latent_store_kernel(LatentShape s, const float *down, uint32_t ldd, uint32_t tokens, uint32_t pos0, const float *w, const float *cos_t,
                                                           const float *sin_t, T *c, T *r) {
    pdl_wait();
    pdl_launch();
    const uint32_t t = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (t >= tokens) return;
    const float *d = down + (size_t)t * ldd;
    const uint32_t pos = pos0 + t, slot = pos % s.rows, half = s.rot_dims / 2;
    float v[32], ss = 0.0f;
#pragma unroll
    for (int j = 0; j < 32; ++j) {
        const uint32_t i = lane + 32 * j;
        v[j] = i < s.kr ? d[i] : 0.0f;
        ss = fmaf(v[j], v[j], ss);
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)s.kr + s.eps);
#pragma unroll
    for (int j = 0; j < 32; ++j) {
        const uint32_t i = lane + 32 * j;
        if (i < s.kr) elem_store(c + (size_t)slot * s.ldc + i, v[j] * inv * w[i]);
    }
    for (uint32_t i = lane; i < s.rot; i += 32)
        elem_store(r + (size_t)slot * s.ldr + i, rot_elem(d + s.kr, i, s.rot_dims, cos_t + (size_t)pos * half, sin_t + (size_t)pos * half));
}

// the shared key part of positions key0 .. out of the ring, in order
template <typename T>
__global__ void __launch_bounds__(256) latent_gather_kernel(LatentShape s, const T *r, T *out, uint32_t key0, uint32_t keys) {
    pdl_wait();
    pdl_launch();
    const uint64_t i = (uint64_t)blockIdx.x * 256 + threadIdx.x;
    if (i >= (uint64_t)keys * s.ldr) return;
    const uint32_t k = (uint32_t)(i / s.ldr), e = (uint32_t)(i - (uint64_t)k * s.ldr);
    out[i] = r[(size_t)((key0 + k) % s.rows) * s.ldr + e];
}

// ---- one token ---------------------------------------------------------------------------------------------------------
// Blocks (h, y): latent columns [128 y, 128 y + 128) of q_lat of head h, scaled; block (h, 0) also the rotated part.
// Block (heads, 0): the token's own row of the ring. qa: [heads][ldq] = [q_lat (kr, padded to ldc) | rotated (ldr)].
template <typename T>
__global__ void __launch_bounds__(256) latent_absorb_kernel(LatentShape s, const float *q, const float *down, const uint16_t *uk, uint32_t ldk, const float *w,
                                                            const float *cos_t, const float *sin_t, T *c, T *r, float *qa, const uint32_t *pos_p) {
    __shared__ float qs[512], part[4][128];
    const uint32_t h = blockIdx.x, tid = threadIdx.x;
    pdl_wait();
    pdl_launch();
    const uint32_t pos = *pos_p, ldq = s.ldc + s.ldr, half = s.rot_dims / 2;
    if (h == s.heads) {
        if (blockIdx.y == 0) store_row<T>(s, down, pos, w, cos_t, sin_t, c, r);
        return;
    }
    const float *qh = q + h * (s.dim + s.rot);
    for (uint32_t i = tid; i < s.dim; i += 256) qs[i] = qh[i] * s.scale;
    if (blockIdx.y == 0)
        for (uint32_t i = tid; i < s.ldr; i += 256)
            qa[(size_t)h * ldq + s.ldc + i] = i < s.rot ? rot_elem(qh + s.dim, i, s.rot_dims, cos_t + (size_t)pos * half, sin_t + (size_t)pos * half) * s.scale : 0.0f;
    __syncthreads();
    const uint32_t cp = tid & 63, grp = tid >> 6, col = blockIdx.y * 128 + 2 * cp;
    float a = 0.0f, b = 0.0f;
    if (col < ldk) {
        const uint16_t *wp = uk + (size_t)h * s.dim * ldk + col;
#pragma unroll 8
        for (uint32_t i = grp; i < s.dim; i += 4) {
            const uint32_t v = *reinterpret_cast<const uint32_t *>(wp + (size_t)i * ldk);
            a = fmaf(qs[i], bf16_lo(v), a);
            b = fmaf(qs[i], bf16_hi(v), b);
        }
    }
    part[grp][2 * cp] = a;
    part[grp][2 * cp + 1] = b;
    __syncthreads();
    if (tid < 128 && blockIdx.y * 128 + tid < s.ldc)
        qa[(size_t)h * ldq + blockIdx.y * 128 + tid] = (part[0][tid] + part[1][tid]) + (part[2][tid] + part[3][tid]);  // (padding: zero weights)
}

constexpr uint32_t PH = 8, PK = 32;  // heads of a block, keys of a tile

// Block (chunk, group): keys [beg + chunk * per, ..) of the window against heads [8 group, 8 group + 8), tiles of 32 keys with
// a running softmax. part: [chunk][heads][ldc + 2] = latent sum, maximum, sum of weights.
template <typename T>
__global__ void __launch_bounds__(256) latent_partial_kernel(LatentShape s, const float *qa, const T *c, const T *r, float *part, uint32_t per, const uint32_t *pos_p) {
    extern __shared__ __align__(16) uint8_t sm_raw[];
    constexpr uint32_t E = 16 / sizeof(T);  // elements of a 16-byte access
    const uint32_t ldq = s.ldc + s.ldr, ldk = ldq + E;  // rows 16 bytes apart in the banks: lanes of a warp read different rows
    float *qs = reinterpret_cast<float *>(sm_raw), *ps = qs + PH * ldq, *st = ps + PH * PK;  // st: [PH] rescale
    T *ks = reinterpret_cast<T *>(st + PH);
    const uint32_t h0 = blockIdx.y * PH, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    pdl_wait();
    pdl_launch();
    const uint32_t pos = *pos_p, beg0 = pos + 1 > s.window ? pos + 1 - s.window : 0u;
    const uint32_t beg = beg0 + blockIdx.x * per, end = min(beg + per, pos + 1), nh = min(PH, s.heads - h0);
    float *out = part + ((size_t)blockIdx.x * s.heads + h0) * (s.ldc + 2);
    if (beg > pos) {
        if (tid < nh) {
            out[(size_t)tid * (s.ldc + 2) + s.ldc] = -INFINITY;
            out[(size_t)tid * (s.ldc + 2) + s.ldc + 1] = 0.0f;
        }
        return;
    }
    for (uint32_t i = tid; i < PH * ldq; i += 256) qs[i] = i < nh * ldq ? qa[(size_t)h0 * ldq + i] : 0.0f;
    float m = -INFINITY, l = 0.0f;  // of head h0 + warp
    // thread: latent columns 2 tid + 512 i and the next one, all heads
    float acc[2][PH][2] = {};
    const uint32_t c16 = s.ldc / E, r16 = s.ldr / E;
    for (uint32_t k0 = beg; k0 < end; k0 += PK) {
        const uint32_t n = min(PK, end - k0);
        __syncthreads();
#pragma unroll
        for (uint32_t i = 0; i < PK / 8; ++i) {  // warp w: keys w, w + 8, ..
            const uint32_t k = warp + 8 * i;
            const size_t slot = (k0 + k) % s.rows;
            for (uint32_t e = lane; e < c16 + r16; e += 32) {
                T *dst = ks + (size_t)k * ldk + e * E;
                const T *src = e < c16 ? c + slot * s.ldc + e * E : r + slot * s.ldr + (e - c16) * E;
                if (k < n) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
                else *reinterpret_cast<uint4 *>(dst) = make_uint4(0, 0, 0, 0);
            }
        }
        asm volatile("cp.async.wait_all;" ::: "memory");
        __syncthreads();
        // scores: warp = head, lane = key
        float sc = 0.0f;
        {
            const T *kp = ks + (size_t)lane * ldk;
            const float *qp = qs + warp * ldq;
            float s1 = 0.0f;
#pragma unroll 4
            for (uint32_t e = 0; e < ldq; e += E) {
                const uint4 kv = *reinterpret_cast<const uint4 *>(kp + e);
                const float4 q0 = *reinterpret_cast<const float4 *>(qp + e);
                if (sizeof(T) == 2) {
                    const float4 q1 = *reinterpret_cast<const float4 *>(qp + e + 4);
                    sc = fmaf(bf16_lo(kv.x), q0.x, sc);
                    s1 = fmaf(bf16_hi(kv.x), q0.y, s1);
                    sc = fmaf(bf16_lo(kv.y), q0.z, sc);
                    s1 = fmaf(bf16_hi(kv.y), q0.w, s1);
                    sc = fmaf(bf16_lo(kv.z), q1.x, sc);
                    s1 = fmaf(bf16_hi(kv.z), q1.y, s1);
                    sc = fmaf(bf16_lo(kv.w), q1.z, sc);
                    s1 = fmaf(bf16_hi(kv.w), q1.w, s1);
                } else {
                    sc = fmaf(__uint_as_float(kv.x), q0.x, sc);
                    s1 = fmaf(__uint_as_float(kv.y), q0.y, s1);
                    sc = fmaf(__uint_as_float(kv.z), q0.z, sc);
                    s1 = fmaf(__uint_as_float(kv.w), q0.w, s1);
                }
            }
            sc += s1;
        }
        if (lane >= n) sc = -INFINITY;
        float mx = sc;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        mx = fmaxf(mx, m);
        const float resc = m == -INFINITY ? 0.0f : expf(m - mx), p = sc == -INFINITY ? 0.0f : expf(sc - mx);
        l = l * resc + warp_sum(p);
        m = mx;
        ps[lane * PH + warp] = p;
        if (lane == 0) st[warp] = resc;
        __syncthreads();
        // latent sums: thread = column pair, all heads
        float rs[PH];
#pragma unroll
        for (uint32_t h = 0; h < PH; ++h) rs[h] = st[h];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const uint32_t col = 2 * tid + 512 * i;
            if (col < s.ldc) {
#pragma unroll
                for (uint32_t h = 0; h < PH; ++h) {
                    acc[i][h][0] *= rs[h];
                    acc[i][h][1] *= rs[h];
                }
#pragma unroll 4
                for (uint32_t k = 0; k < PK; ++k) {
                    float v0, v1;
                    if (sizeof(T) == 2) {
                        const uint32_t v = *reinterpret_cast<const uint32_t *>(ks + (size_t)k * ldk + col);
                        v0 = bf16_lo(v);
                        v1 = bf16_hi(v);
                    } else {
                        const float2 v = *reinterpret_cast<const float2 *>(ks + (size_t)k * ldk + col);
                        v0 = v.x;
                        v1 = v.y;
                    }
                    const float4 pa = *reinterpret_cast<const float4 *>(ps + k * PH), pb = *reinterpret_cast<const float4 *>(ps + k * PH + 4);
                    const float pp[PH] = {pa.x, pa.y, pa.z, pa.w, pb.x, pb.y, pb.z, pb.w};
#pragma unroll
                    for (uint32_t h = 0; h < PH; ++h) {
                        acc[i][h][0] = fmaf(pp[h], v0, acc[i][h][0]);
                        acc[i][h][1] = fmaf(pp[h], v1, acc[i][h][1]);
                    }
                }
            }
        }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const uint32_t col = 2 * tid + 512 * i;
        if (col < s.ldc)
#pragma unroll
            for (uint32_t h = 0; h < PH; ++h)
                if (h < nh) *reinterpret_cast<float2 *>(out + (size_t)h * (s.ldc + 2) + col) = make_float2(acc[i][h][0], acc[i][h][1]);
    }
    if (lane == 0 && warp < nh) {
        out[(size_t)warp * (s.ldc + 2) + s.ldc] = m;
        out[(size_t)warp * (s.ldc + 2) + s.ldc + 1] = l;
    }
}

// Block (h, y): head h's latent sum over all chunks, then value rows [y vper, (y + 1) vper) of the head, gated. A warp takes
// rows warp, warp + 8, ..; the weights of its first four rows (latents up to 512 wide) are asked for ahead of the partial sums.
constexpr uint32_t CR = 4;
__global__ void __launch_bounds__(256) latent_combine_kernel(LatentShape s, const float *part, uint32_t chunks, const uint16_t *uv, uint32_t ldv, const float *gate,
                                                             float *out, uint32_t vper) {
    extern __shared__ __align__(16) float sm[];
    float *o = sm, *wt = sm + s.ldc;  // wt: [chunks]
    const uint32_t h = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const size_t ldp = s.ldc + 2;
    const uint32_t v0 = blockIdx.y * vper + warp, v1 = min(s.vdim, (blockIdx.y + 1) * vper);
    auto weights = [&](uint32_t v, uint32_t c) {
        return v < v1 && c < ldv ? __ldcs(reinterpret_cast<const uint4 *>(uv + (size_t)(h * s.vdim + v) * ldv + c)) : make_uint4(0, 0, 0, 0);
    };
    uint4 pre[CR][2];
#pragma unroll
    for (uint32_t i = 0; i < CR; ++i)
#pragma unroll
        for (uint32_t j = 0; j < 2; ++j) pre[i][j] = weights(v0 + 8 * i, lane * 8 + 256 * j);
    pdl_wait();
    pdl_launch();
    const float *ph = part + (size_t)h * ldp;
    const size_t step = (size_t)s.heads * ldp;
    float m = -INFINITY;
    for (uint32_t k = lane; k < chunks; k += 32) m = fmaxf(m, ph[k * step + s.ldc]);
#pragma unroll
    for (int i = 16; i > 0; i >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, i));
    float l = 0.0f;
    for (uint32_t k = lane; k < chunks; k += 32) {
        const float *p = ph + k * step + s.ldc;
        const float w = p[0] == -INFINITY ? 0.0f : expf(p[0] - m);
        if (warp == 0) wt[k] = w;
        l = fmaf(w, p[1], l);
    }
    l = warp_sum(l);
    __syncthreads();
    const float g = 1.0f / (1.0f + expf(-gate[h])) / l;
    for (uint32_t c = tid; c < s.ldc; c += 256) {
        float a = 0.0f;
        for (uint32_t k0 = 0; k0 < chunks; k0 += 8) {
            float v[8];
#pragma unroll
            for (uint32_t k = 0; k < 8; ++k) v[k] = k0 + k < chunks && wt[k0 + k] > 0.0f ? ph[(k0 + k) * step + c] : 0.0f;  // (an empty chunk wrote no sums)
#pragma unroll
            for (uint32_t k = 0; k < 8; ++k)
                if (k0 + k < chunks) a = fmaf(wt[k0 + k], v[k], a);
        }
        o[c] = a;
    }
    __syncthreads();
    auto dot8 = [&](const uint4 &q, uint32_t c, float a) {
        const float4 x = *reinterpret_cast<const float4 *>(o + c), y = *reinterpret_cast<const float4 *>(o + c + 4);
        a = fmaf(bf16_lo(q.x), x.x, a);
        a = fmaf(bf16_hi(q.x), x.y, a);
        a = fmaf(bf16_lo(q.y), x.z, a);
        a = fmaf(bf16_hi(q.y), x.w, a);
        a = fmaf(bf16_lo(q.z), y.x, a);
        a = fmaf(bf16_hi(q.z), y.y, a);
        a = fmaf(bf16_lo(q.w), y.z, a);
        return fmaf(bf16_hi(q.w), y.w, a);
    };
#pragma unroll
    for (uint32_t i = 0; i < CR; ++i) {
        const uint32_t v = v0 + 8 * i;
        float a = 0.0f;
#pragma unroll
        for (uint32_t j = 0; j < 2; ++j)
            if (lane * 8 + 256 * j < ldv) a = dot8(pre[i][j], lane * 8 + 256 * j, a);
        for (uint32_t c = lane * 8 + 512; c < ldv; c += 256) a = dot8(weights(v, c), c, a);
        a = warp_sum(a);
        if (lane == 0 && v < v1) out[h * s.vdim + v] = a * g;
    }
    for (uint32_t v = v0 + 8 * CR; v < v1; v += 8) {
        float a = 0.0f;
        for (uint32_t c = lane * 8; c < ldv; c += 256) a = dot8(weights(v, c), c, a);
        a = warp_sum(a);
        if (lane == 0) out[h * s.vdim + v] = a * g;
    }
}

}  // namespace

namespace brasa_stack {
namespace {

class LatentAttention : public Mixer {
  public:
    bool configure(const brasa::Json &c, uint32_t width, float eps, std::string &err) override {
        const brasa::Json *mask = c.get("mask"), *rot = c.get("rot");
        if (!mask || !rot) return err = "latent_attention: mask or rot is missing", false;
        double scale = 0.0;
        if (!read_u32(c, "heads", &s_.heads, err) || !read_u32(c, "dim", &s_.dim, err) || !read_u32(c, "rot_dim", &s_.rot, err) ||
            !read_u32(c, "vdim", &s_.vdim, err) || !read_u32(c, "kv_rank", &s_.kr, err) || !read_u32(*mask, "size", &s_.window, err) ||
            !read_u32(*rot, "dims", &s_.rot_dims, err) || !read_f64(*rot, "base", &base_, err) || !read_f64(c, "scale", &scale, err))
            return false;
        if (s_.rot_dims > s_.rot || s_.rot_dims % 2) return err = "latent_attention: rot.dims must be even and at most rot_dim", false;
        if (s_.dim > 512 || s_.vdim > 256 || s_.kr > 1024) return err = "latent_attention: dim up to 512, vdim up to 256, kv_rank up to 1024", false;
        s_.scale = (float)scale;
        s_.eps = eps;
        s_.ldc = up8(s_.kr);
        s_.ldr = up8(s_.rot);
        width_ = width;
        return true;
    }

    int32_t build(Builder &b, const std::string &x) override {
        BRASA_TRY(b.matrix(x + "q", s_.heads * (s_.dim + s_.rot), width_, &q_));
        BRASA_TRY(b.matrix(x + "dkv", s_.kr + s_.rot, width_, &down_));
        BRASA_TRY(b.matrix(x + "uk", s_.heads * s_.dim, s_.kr, &uk_));
        BRASA_TRY(b.matrix(x + "uv", s_.heads * s_.vdim, s_.kr, &uv_));
        BRASA_TRY(b.matrix(x + "g", s_.heads, width_, &g_));
        outs.resize(1);
        BRASA_TRY(b.matrix(x + "o", width_, s_.heads * s_.vdim, &outs[0]));
        BRASA_TRY(b.vector(x + "dkv.norm", s_.kr, &norm_));
        BRASA_TRY(b.rope(base_, s_.rot_dims, &cos_, &sin_));
        const uint64_t t = b.limits.max_tokens, span = std::min<uint64_t>(b.limits.ctx, t + s_.window - 1);
        s_.rows = (uint32_t)((span + 63) / 64 * 64);
        BRASA_TRY(b.get(Builder::STATE, (uint64_t)s_.rows * s_.ldc * b.elem(), &c_));
        BRASA_TRY(b.get(Builder::STATE, (uint64_t)s_.rows * s_.ldr * b.elem(), &r_));
        ldq_ = up8(q_.rows);
        ldd_ = up8(down_.rows);
        ldg_ = up8(s_.heads);
        ldk_ = up8(uk_.rows);
        ldv_ = up8(uv_.rows);
        // one token: keys per block so that the blocks cover the SMs about once
        const uint32_t groups = (s_.heads + PH - 1) / PH, seen = (uint32_t)std::min<uint64_t>(s_.window, b.limits.ctx), tiles = (seen + PK - 1) / PK;
        const uint32_t want = std::max(1u, 148u / groups);
        per_ = PK * ((tiles + want - 1) / want);
        chunks_ = (seen + per_ - 1) / per_;
        Carver c;
        at_.q = c.take(4 * t * ldq_);
        at_.down = c.take(4 * t * ldd_);
        at_.gate = c.take(4 * t * ldg_);
        at_.k = c.take(span * ldk_ * b.elem());
        at_.v = c.take(span * ldv_ * b.elem());
        at_.kr = c.take(span * s_.ldr * b.elem());
        at_.qa = c.take(4ull * s_.heads * (s_.ldc + s_.ldr));
        at_.part = c.take(4ull * chunks_ * s_.heads * (s_.ldc + 2));
        at_.total = c.at;
        return BRASA_OK;
    }

    uint64_t scratch_bytes() const override { return at_.total; }

    void project(const Run &r, std::vector<GemvProblem> &out) override {
        auto add = [&](const Weight &w, uint64_t at, uint32_t ld) {
            GemvProblem g;
            g.p.seg[0] = segment(w, r.h, r.ldh);
            g.p.rows = w.rows;
            g.p.tokens = r.tokens;
            g.p.y = r.scratch + at;
            g.p.ldy = ld;
            out.push_back(g);
        };
        add(q_, at_.q, ldq_);
        add(down_, at_.down, ldd_);
        add(g_, at_.gate, ldg_);
    }

    int32_t mix(const Run &r) override {
        if (r.dev_pos) return r.f32 ? step<float>(r) : step<__nv_bfloat16>(r);
        return r.f32 ? run<float>(r) : run<__nv_bfloat16>(r);
    }

  private:
    template <typename T>
    int32_t run(const Run &r) {
        brasa_ctx *ctx = r.cmd->ctx;
        auto f = [&](uint64_t at) { return (float *)(r.scratch + at); };
        T *c = (T *)c_, *kr = (T *)r_, *krow = (T *)(r.scratch + at_.kr);
        BRASA_CUDA(ctx, brasa_launch_dependent(ctx, latent_store_kernel<T>, dim3((r.tokens + 7) / 8), dim3(256), 0, s_, f(at_.down), ldd_, r.tokens, r.pos0, norm_, cos_, sin_, c, kr));
        BRASA_TRY(brasa_post_launch(r.cmd, "latent_store"));
        // every position some query of the run sees, in order; the ring holds them in at most two pieces
        const uint32_t key0 = r.pos0 + 1 > s_.window ? r.pos0 + 1 - s_.window : 0u, keys = r.pos0 + r.tokens - key0;
        BRASA_CUDA(ctx, brasa_launch_dependent(ctx, latent_gather_kernel<T>, dim3((unsigned)(((uint64_t)keys * s_.ldr + 255) / 256)), dim3(256), 0, s_, kr, krow, key0, keys));
        BRASA_TRY(brasa_post_launch(r.cmd, "latent_gather"));
        LinearProblem lp[4];
        uint32_t n = 0;
        for (uint32_t done = 0; done < keys;) {
            const uint32_t slot = (key0 + done) % s_.rows, len = std::min(keys - done, s_.rows - slot);
            for (int kv = 0; kv < 2; ++kv) {
                const Weight &w = kv ? uv_ : uk_;
                const uint32_t ld = kv ? ldv_ : ldk_;
                LinearProblem &p = lp[n++];
                p.seg[0] = segment(w, c + (size_t)slot * s_.ldc, s_.ldc);
                p.rows = w.rows;
                p.tokens = len;
                p.y = (T *)(r.scratch + (kv ? at_.v : at_.k)) + (size_t)done * ld;
                p.ldy = ld;
                p.y_bf16 = sizeof(T) == 2;
            }
            done += len;
        }
        BRASA_TRY(brasa_linear_launch(r.cmd, lp, n, r.f32));
        WindowAttn a{};
        a.q = f(at_.q);
        a.k = r.scratch + at_.k;
        a.v = r.scratch + at_.v;
        a.kr = krow;
        a.cos_t = cos_;
        a.sin_t = sin_;
        a.gate = f(at_.gate);
        a.out = r.out[0];
        a.ldq = ldq_; a.ldk = ldk_; a.ldv = ldv_; a.ldr = s_.ldr; a.ldg = ldg_; a.ldo = r.ldo[0];
        a.tokens = r.tokens; a.heads = s_.heads; a.dim = s_.dim; a.rot = s_.rot; a.rot_dims = s_.rot_dims; a.vdim = s_.vdim;
        a.pos0 = r.pos0; a.key0 = key0; a.keys = keys; a.window = s_.window;
        a.scale = s_.scale;
        a.kv_heads = s_.heads; a.kstep = s_.dim; a.vstep = s_.vdim;
        a.out_scale = 1.0f;
        return brasa_window_attention_launch(r.cmd, a, r.f32);
    }

    template <typename T>
    int32_t step(const Run &r) {
        brasa_ctx *ctx = r.cmd->ctx;
        auto f = [&](uint64_t at) { return (float *)(r.scratch + at); };
        T *c = (T *)c_, *kr = (T *)r_;
        BRASA_CUDA(ctx, brasa_launch_dependent(ctx, latent_absorb_kernel<T>, dim3(s_.heads + 1, (s_.ldc + 127) / 128), dim3(256), 0, s_, f(at_.q), f(at_.down), uk_.p, uk_.ld,
                                               norm_, cos_, sin_, c, kr, f(at_.qa), r.dev_pos));
        BRASA_TRY(brasa_post_launch(r.cmd, "latent_absorb"));
        const uint32_t ldq = s_.ldc + s_.ldr;
        const size_t smem = (size_t)(PH * ldq + PH * PK + PH) * 4 + (size_t)PK * (ldq + 16 / sizeof(T)) * sizeof(T);
        BRASA_REQUIRE(ctx, smem + 1024 <= ctx->smem_optin, "latent attention: latent too wide");
        BRASA_TRY(brasa_smem_optin(ctx, (const void *)latent_partial_kernel<T>, smem));
        BRASA_CUDA(ctx, brasa_launch_dependent(ctx, latent_partial_kernel<T>, dim3(chunks_, (s_.heads + PH - 1) / PH), dim3(256), smem, s_, f(at_.qa), c, kr, f(at_.part), per_,
                                               r.dev_pos));
        BRASA_TRY(brasa_post_launch(r.cmd, "latent_partial"));
        const uint32_t split = std::max(1u, std::min((s_.vdim + 7) / 8, 148u / s_.heads)), vper = (s_.vdim + split - 1) / split;
        const size_t csm = (size_t)(s_.ldc + chunks_) * 4;
        BRASA_TRY(brasa_smem_optin(ctx, (const void *)latent_combine_kernel, std::max<size_t>(csm, 48 * 1024)));
        BRASA_CUDA(ctx, brasa_launch_dependent(ctx, latent_combine_kernel, dim3(s_.heads, (s_.vdim + vper - 1) / vper), dim3(256), csm, s_, f(at_.part), chunks_, uv_.p, uv_.ld,
                                               f(at_.gate), (float *)r.out[0], vper));
        return brasa_post_launch(r.cmd, "latent_combine");
    }

    LatentShape s_{};
    double base_ = 0.0;
    uint32_t width_ = 0, ldq_ = 0, ldd_ = 0, ldg_ = 0, ldk_ = 0, ldv_ = 0, per_ = 0, chunks_ = 0;
    Weight q_, down_, uk_, uv_, g_;
    const float *norm_ = nullptr, *cos_ = nullptr, *sin_ = nullptr;
    void *c_ = nullptr, *r_ = nullptr;
    struct {
        uint64_t q, down, gate, k, v, kr, qa, part, total;
    } at_{};
};

}  // namespace

std::unique_ptr<Mixer> make_latent_attention() { return std::unique_ptr<Mixer>(new LatentAttention()); }

}  // namespace brasa_stack
