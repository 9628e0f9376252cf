// Grouped-query attention inside a sliding window, with rotary positions on the first dimensions of each head and softcapped
// scores: the left side of "parallel". Query heads h, h + 1, .. of a group share one key / value head.
//
// Cache: rings of key rows (rotated) and value rows, position p in row p % rows, rows >= window - 1 + the longest run (a run's
// own tokens never push out what its first query still sees) and a multiple of 128, so that a 128-key tile of window_attn.cu is
// contiguous. Heads lie up8(dim) and up8(vdim) elements apart. The rings are cleared once: tiles read rows nothing was stored in.
// Many tokens: attn_store_kernel, then window_attn.cu over the rings as they are.
// One token: attn_step_kernel, one cluster of blocks per key head (and per eight of its query heads), the keys dealt out to the
// cluster's warps eight at a time, each warp with softmax sums of its own, merged through distributed shared memory.
#include <cooperative_groups.h>
#include <cuda_bf16.h>

#include "conv_device.cuh"
#include "stack.h"
#include "tc_device.cuh"
#include "window_attn.h"

using namespace brasa_dev;
namespace cg = cooperative_groups;

namespace {

struct AttnShape {
    uint32_t heads, kv_heads, dim, vdim, rot_dims, window;
    uint32_t rows, kstep, vstep;  // the rings
    float scale, softcap, out_scale;
};

// element e of a head whose first `dims` entries are rotated by the angles in c and s
__device__ __forceinline__ float rot_elem(const float *x, uint32_t e, uint32_t dims, const float *c, const float *s) {
    const uint32_t half = dims / 2;
    if (e < half) return x[e] * c[e] - x[e + half] * s[e];
    if (e < dims) return x[e] * c[e - half] + x[e - half] * s[e - half];
    return x[e];
}

// Keys and values of a run into the rings; one warp per (token, key head).
template <typename T>
__global__ void __launch_bounds__(256) attn_store_kernel(AttnShape s, const float *k, uint32_t ldk, const float *v, uint32_t ldv, uint32_t tokens, uint32_t pos0,
                                                         const float *cos_t, const float *sin_t, T *kc, T *vc) {
    pdl_wait();
    pdl_launch();
    const uint32_t i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (i >= tokens * s.kv_heads) return;
    const uint32_t t = i / s.kv_heads, g = i - t * s.kv_heads, pos = pos0 + t, half = s.rot_dims / 2;
    const size_t slot = pos % s.rows;
    const float *kr = k + (size_t)t * ldk + g * s.dim, *vr = v + (size_t)t * ldv + g * s.vdim;
    for (uint32_t e = lane; e < s.dim; e += 32)
        elem_store(kc + (slot * s.kv_heads + g) * s.kstep + e, rot_elem(kr, e, s.rot_dims, cos_t + (size_t)pos * half, sin_t + (size_t)pos * half));
    for (uint32_t e = lane; e < s.vdim; e += 32) elem_store(vc + (slot * s.kv_heads + g) * s.vstep + e, vr[e]);
}

constexpr uint32_t PH = 8, PW = 16, PK = 8, VMAX = 8;  // query heads of a block, warps of a block, keys of a tile, value columns of a lane (vdim up to 256)

// Shared memory of a step's block, in floats: parts [PW][heads][ldp] and the block's merged sums [heads][ldp] (ldp: value columns,
// then maximum and sum of weights), weights of the parts [heads][PW], rotated queries [heads][kstep], this token's key and value.
struct StepPlan {
    uint32_t heads, ldp, own, wt, qs, now, bytes;
    __host__ __device__ StepPlan(const AttnShape &s, uint32_t elem) {
        const uint32_t share = s.heads / s.kv_heads;
        heads = share < PH ? share : PH;
        ldp = s.vdim + 2;
        own = PW * heads * ldp;
        wt = own + heads * ldp;
        qs = (wt + heads * PW + 3) / 4 * 4;
        now = qs + heads * s.kstep;
        bytes = now * 4 + (s.kstep + s.vstep) * elem;
    }
};

// Grid (splits, groups): cluster = one group's splits; group = key head g and its query heads [8 sub, 8 sub + 8). A tile of eight
// keys: lane = key lane / 4 and every fourth 16-byte piece of its row from piece lane % 4 on; then value columns lane, lane + 32, ..
// V: value columns of a lane; HM: the most query heads of a block.
template <typename T, int V, uint32_t HM>
__global__ void __launch_bounds__(32 * PW, 1) attn_step_kernel(AttnShape s, const float *q, const float *k, const float *v, const float *cos_t, const float *sin_t, T *kc,
                                                               T *vc, float *out, const uint32_t *pos_p) {
    extern __shared__ __align__(16) float sm[];
    constexpr uint32_t E = 16 / sizeof(T);  // elements of a 16-byte access
    const StepPlan pl(s, sizeof(T));
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, splits = gridDim.x, rank = blockIdx.x;
    const uint32_t share = s.heads / s.kv_heads, subs = (share + PH - 1) / PH, g = blockIdx.y / subs, h0 = g * share + blockIdx.y % subs * PH;
    const uint32_t nh = min(PH, (g + 1) * share - h0), ldp = pl.ldp, half = s.rot_dims / 2;
    float *parts = sm, *own = sm + pl.own, *wt = sm + pl.wt, *qs = sm + pl.qs;
    T *k_now = reinterpret_cast<T *>(sm + pl.now), *v_now = k_now + s.kstep;
    // The position and the older keys and values were written several kernels ago: the first tile is asked for ahead of the wait.
    const uint32_t pos = *pos_p, beg = pos + 1 > s.window ? pos + 1 - s.window : 0u, slot0 = beg % s.rows;
    const float *ct = cos_t + (size_t)pos * half, *st = sin_t + (size_t)pos * half;
    auto slot_of = [&](uint32_t key) {  // of a visible position
        const uint32_t r = slot0 + key - beg;
        return (size_t)(r >= s.rows ? r - s.rows : r) * s.kv_heads + g;
    };
    constexpr uint32_t KR = 4;  // 16-byte pieces of a lane's key kept ahead
    uint4 kk4[KR];
    float vv[PK][V];
    auto load = [&](uint32_t t0) {  // positions before this token's
        const uint32_t key = t0 + (lane >> 2);
        const T *kp = kc + slot_of(key < pos ? key : beg) * s.kstep;
#pragma unroll
        for (uint32_t i = 0; i < KR; ++i) {
            const uint32_t e = ((lane & 3) + 4 * i) * E;
            kk4[i] = key < pos && e < s.kstep ? *reinterpret_cast<const uint4 *>(kp + e) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
        for (uint32_t j = 0; j < PK; ++j) {
            const T *vp = vc + slot_of(t0 + j < pos ? t0 + j : beg) * s.vstep;
#pragma unroll
            for (int c = 0; c < V; ++c) vv[j][c] = t0 + j < pos && lane + 32 * c < s.vdim ? elem_load(vp + lane + 32 * c) : 0.0f;
        }
    };
    const uint32_t first = beg + PK * (rank * PW + warp);
    load(first);
    pdl_wait();
    pdl_launch();
    const bool keeper = rank == 0 && blockIdx.y % subs == 0;  // stores this token's rows (nobody reads them there in this step)
    for (uint32_t i = warp; i < nh + 2; i += PW) {
        if (i < nh) {
            for (uint32_t e = lane; e < s.kstep; e += 32) qs[i * s.kstep + e] = e < s.dim ? rot_elem(q + (size_t)(h0 + i) * s.dim, e, s.rot_dims, ct, st) * s.scale : 0.0f;
        } else {
            const bool key = i == nh;
            const uint32_t n = key ? s.dim : s.vdim, step = key ? s.kstep : s.vstep;
            T *now = key ? k_now : v_now, *keep = (key ? kc : vc) + slot_of(pos) * step;
            for (uint32_t e = lane; e < step; e += 32) {
                elem_store(now + e, e >= n ? 0.0f : (key ? rot_elem(k + g * s.dim, e, s.rot_dims, ct, st) : v[g * s.vdim + e]));
                if (keeper && e < n) keep[e] = now[e];
            }
        }
    }
    __syncthreads();
    float m[HM], l[HM], acc[HM][V];
#pragma unroll
    for (uint32_t h = 0; h < HM; ++h) {
        m[h] = -INFINITY;
        l[h] = 0.0f;
#pragma unroll
        for (int c = 0; c < V; ++c) acc[h][c] = 0.0f;
    }
    for (uint32_t t0 = first; t0 <= pos; t0 += PK * PW * splits) {
        const uint32_t key = t0 + (lane >> 2);
        const bool live = key <= pos;
        const T *kp = key >= pos ? k_now : kc + slot_of(key) * s.kstep;
        if (t0 != first) load(t0);
        if (key == pos)
#pragma unroll
            for (uint32_t i = 0; i < KR; ++i)
                if (((lane & 3) + 4 * i) * E < s.kstep) kk4[i] = *reinterpret_cast<const uint4 *>(k_now + ((lane & 3) + 4 * i) * E);
#pragma unroll
        for (uint32_t j = 0; j < PK; ++j)
            if (t0 + j == pos)
#pragma unroll
                for (int c = 0; c < V; ++c) vv[j][c] = lane + 32 * c < s.vdim ? elem_load(v_now + lane + 32 * c) : 0.0f;
        float sc[HM];
#pragma unroll
        for (uint32_t h = 0; h < HM; ++h) sc[h] = 0.0f;
        auto dots = [&](const uint4 &kv, uint32_t e) {
            float kk[E];
            if (sizeof(T) == 2) {
                kk[0] = bf16_lo(kv.x); kk[1] = bf16_hi(kv.x); kk[2] = bf16_lo(kv.y); kk[3] = bf16_hi(kv.y);
                kk[E - 4] = bf16_lo(kv.z); kk[E - 3] = bf16_hi(kv.z); kk[E - 2] = bf16_lo(kv.w); kk[E - 1] = bf16_hi(kv.w);
            } else {
                kk[0] = __uint_as_float(kv.x); kk[1] = __uint_as_float(kv.y); kk[2] = __uint_as_float(kv.z); kk[3] = __uint_as_float(kv.w);
            }
#pragma unroll
            for (uint32_t h = 0; h < HM; ++h)
                if (h < nh)
#pragma unroll
                    for (uint32_t i = 0; i < E; i += 4) {
                        const float4 qv = *reinterpret_cast<const float4 *>(qs + h * s.kstep + e + i);
                        sc[h] = fmaf(kk[i], qv.x, fmaf(kk[i + 1], qv.y, fmaf(kk[i + 2], qv.z, fmaf(kk[i + 3], qv.w, sc[h]))));
                    }
        };
#pragma unroll
        for (uint32_t i = 0; i < KR; ++i)
            if (((lane & 3) + 4 * i) * E < s.kstep) dots(kk4[i], ((lane & 3) + 4 * i) * E);
        for (uint32_t e = ((lane & 3) + 4 * KR) * E; e < s.kstep; e += 4 * E) dots(*reinterpret_cast<const uint4 *>(kp + e), e);
#pragma unroll
        for (uint32_t h = 0; h < HM; ++h)
            if (h < nh) {
                float x = sc[h];
                x += __shfl_xor_sync(0xffffffffu, x, 1);
                x += __shfl_xor_sync(0xffffffffu, x, 2);
                if (s.softcap > 0.0f) x = s.softcap * tanhf(x / s.softcap);
                if (!live) x = -INFINITY;
                float mx = x;
#pragma unroll
                for (int o = 16; o > 2; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
                mx = fmaxf(mx, m[h]);  // finite: a tile has at least one visible key
                float p = expf(x - mx), r = expf(m[h] - mx);
                m[h] = mx;
#pragma unroll
                for (int c = 0; c < V; ++c) acc[h][c] *= r;
                l[h] *= r;
#pragma unroll
                for (uint32_t j = 0; j < PK; ++j) {
                    const float w = __shfl_sync(0xffffffffu, p, 4 * j);
                    l[h] += w;
#pragma unroll
                    for (int c = 0; c < V; ++c) acc[h][c] = fmaf(w, vv[j][c], acc[h][c]);
                }
            }
    }
#pragma unroll
    for (uint32_t h = 0; h < HM; ++h)
        if (h < nh) {
            float *p = parts + (warp * pl.heads + h) * ldp;
#pragma unroll
            for (int c = 0; c < V; ++c)
                if (lane + 32 * c < s.vdim) p[lane + 32 * c] = acc[h][c];
            if (lane == 0) {
                p[s.vdim] = m[h];
                p[s.vdim + 1] = l[h];
            }
        }
    __syncthreads();
    // The block's sums: head `warp`, lane = part; then all columns. (A warp that had no tile: maximum -inf, weight 0.)
    if (warp < nh) {
        const float *p = parts + (lane * pl.heads + warp) * ldp + s.vdim;
        const float f = lane < PW ? p[0] : -INFINITY;
        float mx = f;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        const float r = f == -INFINITY ? 0.0f : expf(f - mx);
        if (lane < PW) wt[warp * PW + lane] = r;
        const float ls = warp_sum(lane < PW ? r * p[1] : 0.0f);
        if (lane == 0) {
            own[warp * ldp + s.vdim] = mx;
            own[warp * ldp + s.vdim + 1] = ls;
        }
    }
    __syncthreads();
    for (uint32_t h = 0; h < nh; ++h)
        for (uint32_t e = tid; e < s.vdim; e += 32 * PW) {
            float a = 0.0f;
#pragma unroll
            for (uint32_t w = 0; w < PW; ++w) a = fmaf(wt[h * PW + w], parts[(w * pl.heads + h) * ldp + e], a);
            own[h * ldp + e] = a;
        }
    cg::cluster_group cluster = cg::this_cluster();
    cluster.sync();
    // The cluster's sums: block `rank` takes heads rank, rank + splits, ..
    for (uint32_t h = rank; h < nh; h += splits) {
        float mx = -INFINITY, ls = 0.0f, r[8];
#pragma unroll
        for (uint32_t b = 0; b < 8; ++b) {
            r[b] = b < splits ? cluster.map_shared_rank(own, b)[h * ldp + s.vdim] : -INFINITY;
            mx = fmaxf(mx, r[b]);
        }
#pragma unroll
        for (uint32_t b = 0; b < 8; ++b) {
            r[b] = r[b] == -INFINITY ? 0.0f : expf(r[b] - mx);
            if (b < splits) ls = fmaf(r[b], cluster.map_shared_rank(own, b)[h * ldp + s.vdim + 1], ls);
        }
        for (uint32_t e = tid; e < s.vdim; e += 32 * PW) {
            float a = 0.0f;
#pragma unroll
            for (uint32_t b = 0; b < 8; ++b)
                if (b < splits) a = fmaf(r[b], cluster.map_shared_rank(own, b)[h * ldp + e], a);
            out[(size_t)(h0 + h) * s.vdim + e] = a / ls * s.out_scale;
        }
    }
    cluster.sync();  // nobody leaves while its sums are being read
}

}  // namespace

namespace brasa_stack {
namespace {

class WindowAttention : public Mixer {
  public:
    bool configure(const brasa::Json &c, uint32_t width, float, std::string &err) override {
        const brasa::Json *mask = c.get("mask"), *rot = c.get("rot");
        if (!mask || !rot) return err = "attention: mask or rot is missing", false;
        double scale = 0.0, cap = 0.0;
        if (!read_u32(c, "heads", &s_.heads, err) || !read_u32(c, "kv_heads", &s_.kv_heads, err) || !read_u32(c, "dim", &s_.dim, err) ||
            !read_u32(c, "vdim", &s_.vdim, err) || !read_u32(*mask, "size", &s_.window, err) || !read_u32(*rot, "dims", &s_.rot_dims, err) ||
            !read_f64(*rot, "base", &base_, err) || !read_f64(c, "scale", &scale, err) || !read_f64(c, "softcap", &cap, err))
            return false;
        if (s_.heads % s_.kv_heads) return err = "attention: heads must be a multiple of kv_heads", false;
        if (s_.rot_dims > s_.dim || s_.rot_dims % 2) return err = "attention: rot.dims must be even and at most dim", false;
        if (s_.dim > 512 || s_.vdim > 32 * VMAX) return err = "attention: dim up to 512, vdim up to 256", false;
        if (!(cap > 0.0)) return err = "attention: softcap must be positive", false;
        s_.scale = (float)scale;
        s_.softcap = (float)cap;
        s_.out_scale = 1.0f;
        s_.kstep = up8(s_.dim);
        s_.vstep = up8(s_.vdim);
        width_ = width;
        return true;
    }
    bool scale_output(float f) override {
        s_.out_scale = f;
        return true;
    }

    int32_t build(Builder &b, const std::string &x) override {
        BRASA_TRY(b.matrix(x + "q", s_.heads * s_.dim, width_, &q_));
        BRASA_TRY(b.matrix(x + "k", s_.kv_heads * s_.dim, width_, &k_));
        BRASA_TRY(b.matrix(x + "v", s_.kv_heads * s_.vdim, width_, &v_));
        outs.resize(1);
        BRASA_TRY(b.matrix(x + "o", width_, s_.heads * s_.vdim, &outs[0]));
        BRASA_TRY(b.rope(base_, s_.rot_dims, &cos_, &sin_));
        const uint64_t t = b.limits.max_tokens, span = std::min<uint64_t>(b.limits.ctx, t + s_.window - 1);
        s_.rows = (uint32_t)((span + 127) / 128 * 128);
        const uint64_t kn = (uint64_t)s_.rows * s_.kv_heads * s_.kstep * b.elem(), vn = (uint64_t)s_.rows * s_.kv_heads * s_.vstep * b.elem();
        BRASA_TRY(b.get(Builder::STATE, kn, &kc_));
        BRASA_TRY(b.get(Builder::STATE, vn, &vc_));
        if (b.m) {
            BRASA_CUDA(b.m->ctx, cudaMemsetAsync(kc_, 0, kn, b.m->ctx->stream));
            BRASA_CUDA(b.m->ctx, cudaMemsetAsync(vc_, 0, vn, b.m->ctx->stream));
        }
        seen_ = (uint32_t)std::min<uint64_t>(s_.window, b.limits.ctx);
        ldq_ = up8(q_.rows);
        ldk_ = up8(k_.rows);
        ldv_ = up8(v_.rows);
        Carver c;
        at_.q = c.take(4 * t * ldq_);
        at_.k = c.take(4 * t * ldk_);
        at_.v = c.take(4 * t * ldv_);
        at_.total = c.at;
        return BRASA_OK;
    }

    uint64_t scratch_bytes() const override { return at_.total; }

    void project(const Run &r, std::vector<GemvProblem> &out) override {
        add_projection(r, q_, at_.q, ldq_, out);
        add_projection(r, k_, at_.k, ldk_, out);
        add_projection(r, v_, at_.v, ldv_, out);
    }

    int32_t mix(const Run &r) override {
        if (r.dev_pos) return r.f32 ? step_as<float>(r) : step_as<__nv_bfloat16>(r);
        return r.f32 ? run<float>(r) : run<__nv_bfloat16>(r);
    }

  private:
    template <typename T>
    int32_t run(const Run &r) {
        brasa_ctx *ctx = r.cmd->ctx;
        auto f = [&](uint64_t at) { return (const float *)(r.scratch + at); };
        BRASA_CUDA(ctx, brasa_launch_dependent(ctx, attn_store_kernel<T>, dim3((r.tokens * s_.kv_heads + 7) / 8), dim3(256), 0, s_, f(at_.k), ldk_, f(at_.v), ldv_, r.tokens,
                                               r.pos0, cos_, sin_, (T *)kc_, (T *)vc_));
        BRASA_TRY(brasa_post_launch(r.cmd, "attn_store"));
        WindowAttn a{};
        a.q = f(at_.q);
        a.k = kc_;
        a.v = vc_;
        a.cos_t = cos_;
        a.sin_t = sin_;
        a.out = r.out[0];
        a.ldq = ldq_; a.ldk = s_.kv_heads * s_.kstep; a.ldv = s_.kv_heads * s_.vstep; a.ldo = r.ldo[0];
        a.tokens = r.tokens; a.heads = s_.heads; a.dim = s_.dim; a.rot_dims = s_.rot_dims; a.vdim = s_.vdim;
        a.pos0 = r.pos0;
        a.key0 = (r.pos0 + 1 > s_.window ? r.pos0 + 1 - s_.window : 0u) / 128 * 128;
        a.keys = r.pos0 + r.tokens - a.key0;
        a.window = s_.window;
        a.scale = s_.scale;
        a.kv_heads = s_.kv_heads; a.kstep = s_.kstep; a.vstep = s_.vstep;
        a.ring = s_.rows;
        a.softcap = s_.softcap;
        a.out_scale = s_.out_scale;
        return brasa_window_attention_launch(r.cmd, a, r.f32);
    }

    template <typename T>
    int32_t step_as(const Run &r) {
        const bool few = s_.heads / s_.kv_heads <= 4;
        if (s_.vdim <= 64) return few ? step<T, 2, 4>(r) : step<T, 2, PH>(r);
        if (s_.vdim <= 128) return few ? step<T, 4, 4>(r) : step<T, 4, PH>(r);
        return few ? step<T, (int)VMAX, 4>(r) : step<T, (int)VMAX, PH>(r);
    }
    template <typename T, int V, uint32_t HM>
    int32_t step(const Run &r) {
        brasa_ctx *ctx = r.cmd->ctx;
        auto f = [&](uint64_t at) { return (const float *)(r.scratch + at); };
        const uint32_t share = s_.heads / s_.kv_heads, groups = s_.kv_heads * ((share + PH - 1) / PH);
        uint32_t splits = 1;  // a cluster of at most eight blocks, no more than there are tiles for
        while (splits < 8 && splits * PK * PW < seen_) splits *= 2;
        const size_t smem = StepPlan(s_, sizeof(T)).bytes;
        BRASA_REQUIRE(ctx, smem + 1024 <= ctx->smem_optin, "attention: head sizes too large");
        auto kernel = attn_step_kernel<T, V, HM>;
        BRASA_TRY(brasa_smem_optin(ctx, (const void *)kernel, std::max<size_t>(smem, 48 * 1024)));
        cudaLaunchConfig_t cfg{};
        cfg.gridDim = dim3(splits, groups);
        cfg.blockDim = dim3(32 * PW);
        cfg.dynamicSmemBytes = smem;
        cfg.stream = ctx->stream;
        cudaLaunchAttribute attr[2];
        attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[0].val.programmaticStreamSerializationAllowed = ctx->pdl ? 1 : 0;
        attr[1].id = cudaLaunchAttributeClusterDimension;
        attr[1].val.clusterDim.x = splits;
        attr[1].val.clusterDim.y = attr[1].val.clusterDim.z = 1;
        cfg.attrs = attr;
        cfg.numAttrs = 2;
        BRASA_CUDA(ctx, cudaLaunchKernelEx(&cfg, kernel, s_, f(at_.q), f(at_.k), f(at_.v), cos_, sin_, (T *)kc_, (T *)vc_, (float *)r.out[0], r.dev_pos));
        return brasa_post_launch(r.cmd, "attn_step");
    }

    AttnShape s_{};
    double base_ = 0.0;
    uint32_t width_ = 0, seen_ = 0, ldq_ = 0, ldk_ = 0, ldv_ = 0;
    Weight q_, k_, v_;
    const float *cos_ = nullptr, *sin_ = nullptr;
    void *kc_ = nullptr, *vc_ = nullptr;
    struct {
        uint64_t q, k, v, total;
    } at_{};
};

}  // namespace

std::unique_ptr<Mixer> make_window_attention() { return std::unique_ptr<Mixer>(new WindowAttention()); }

}  // namespace brasa_stack
