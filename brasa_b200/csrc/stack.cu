// Layer-stack models (stack.h): the configuration reader, weights, workspace, the layer loop for runs of tokens and for one
// token, and the families built on it.
//
// Dunuzen (Wiring::BRANCHES): a layer adds its mixer's and its feed-forward's result to the residual stream, each computed from
// the same x behind a layer norm of its own; the feed-forward is two biased products with a squared relu between them. Both
// branches read the same x, so one pass over x forms both norms, the mixer's projections and the feed-forward's first product go
// into one launch, and the output projection and the feed-forward's second product are one product over the concatenation of
// their inputs that adds to x in its epilogue.
//
// Gugedra (Wiring::SANDWICH): a sublayer's input and its result are RMS-normed, one sublayer behind the other, and a small gated
// input per token and layer follows. Many tokens: one pass over a row norms a result, adds it and norms the next input; the
// gated feed-forward's and the token side's products form their activations in the epilogue. One token: the norm and the addition
// are formed by every block of the next product on its way in, so a layer is its products and its mixer, nothing else.
#include "stack.h"

#include <cuda_bf16.h>
#include <math.h>

#include "stack_model.h"
#include "tc_device.cuh"

using namespace brasa_dev;

int32_t brasa_argmax_launch(brasa_cmd *cmd, const float *logits, uint32_t n, uint32_t *out);

namespace brasa_stack {

bool read_u32(const brasa::Json &c, const char *key, uint32_t *out, std::string &err) {
    const brasa::Json *j = c.get(key);
    if (!j || j->kind != brasa::Json::Num || !j->is_int || j->inum <= 0 || j->inum > 0x7fffffff) return err = std::string("config.json: ") + key + " is missing or out of range", false;
    *out = (uint32_t)j->inum;
    return true;
}
bool read_f64(const brasa::Json &c, const char *key, double *out, std::string &err) {
    const brasa::Json *j = c.get(key);
    if (!j || j->kind != brasa::Json::Num) return err = std::string("config.json: ") + key + " is missing", false;
    *out = j->num;
    return true;
}

// ---- Builder -----------------------------------------------------------------------------------------------------------
namespace {

__global__ void widen_bf16_kernel(const uint16_t *src, float *dst, uint64_t n) {
    const uint64_t i = (uint64_t)blockIdx.x * 256 + threadIdx.x;
    if (i < n) dst[i] = __uint_as_float((uint32_t)src[i] << 16);
}
__global__ void pad_rows_kernel(const uint16_t *src, uint16_t *dst, uint32_t rows, uint32_t cols, uint32_t ld) {
    const uint64_t i = (uint64_t)blockIdx.x * 256 + threadIdx.x;
    if (i >= (uint64_t)rows * ld) return;
    const uint32_t r = (uint32_t)(i / ld), c = (uint32_t)(i - (uint64_t)r * ld);
    dst[i] = c < cols ? src[(size_t)r * cols + c] : (uint16_t)0;
}

// row r of a matrix to row r of the first (second: 1) kind of alternating blocks of 32 rows
__global__ void interleave_rows_kernel(const uint16_t *src, uint16_t *dst, uint32_t rows, uint32_t cols, uint32_t ld, uint32_t second) {
    const uint64_t i = (uint64_t)blockIdx.x * 256 + threadIdx.x;
    if (i >= (uint64_t)rows * ld) return;
    const uint32_t r = (uint32_t)(i / ld), c = (uint32_t)(i - (uint64_t)r * ld);
    dst[(size_t)((r >> 5) * 64 + second * 32 + (r & 31)) * ld + c] = c < cols ? src[(size_t)r * cols + c] : (uint16_t)0;
}

std::string shape_text(const std::vector<uint64_t> &s) {
    std::string t = "[";
    for (size_t i = 0; i < s.size(); ++i) t += (i ? ", " : "") + std::to_string(s[i]);
    return t + "]";
}

}  // namespace

int32_t Builder::fail(const std::string &what) {
    err = what;
    return m ? brasa_fail(m->ctx, BRASA_EIO, "%s", what.c_str()) : BRASA_EIO;
}

int32_t Builder::get(Class c, uint64_t n, void **out) {
    bytes[c] += brasa_plan_buffer_bytes(n);
    if (!m) {
        *out = nullptr;
        return BRASA_OK;
    }
    brasa_buf *b;
    BRASA_TRY(brasa_buf_alloc(m->ctx, n, &b));
    m->owned.push_back(b);
    *out = b->ptr;
    return BRASA_OK;
}

int32_t Builder::matrix(const std::string &name, uint32_t rows, uint32_t cols, Weight *out) {
    const brasa::TensorInfo *t = file->tensor(name);
    if (!t) return fail("missing tensor " + name);
    if (t->dtype != "bf16" || t->shape.size() != 2 || (rows && t->shape[0] != rows) || (cols && t->shape[1] != cols) || t->shape[0] == 0 || t->shape[1] == 0)
        return fail(name + ": unexpected type or shape " + shape_text(t->shape));
    out->rows = (uint32_t)t->shape[0];
    out->cols = (uint32_t)t->shape[1];
    out->ld = up8(out->cols);
    void *p;
    const uint64_t n = (uint64_t)out->rows * out->ld;
    BRASA_TRY(get(WEIGHTS, n * 2, &p));
    out->p = (const uint16_t *)p;
    if (!m) return BRASA_OK;
    if (out->ld == out->cols) return brasa_stage_upload(m, p, *file, *t);
    BRASA_TRY(brasa_stage_upload(m, staging->ptr, *file, *t));
    pad_rows_kernel<<<(unsigned)((n + 255) / 256), 256, 0, m->ctx->stream>>>((const uint16_t *)staging->ptr, (uint16_t *)p, out->rows, out->cols, out->ld);
    return brasa_post_launch(cmd, "pad_rows");
}

int32_t Builder::interleaved(const std::string &first, const std::string &second, uint32_t rows, uint32_t cols, Weight *out) {
    out->rows = (rows + 31) / 32 * 64;
    out->cols = cols;
    out->ld = up8(cols);
    void *p;
    const uint64_t n = (uint64_t)out->rows * out->ld * 2;
    BRASA_TRY(get(WEIGHTS, n, &p));
    out->p = (const uint16_t *)p;
    if (m) BRASA_CUDA(m->ctx, cudaMemsetAsync(p, 0, n, m->ctx->stream));
    for (int i = 0; i < 2; ++i) {
        const std::string &name = i ? second : first;
        const brasa::TensorInfo *t = file->tensor(name);
        if (!t) return fail("missing tensor " + name);
        if (t->dtype != "bf16" || t->shape.size() != 2 || t->shape[0] != rows || t->shape[1] != cols) return fail(name + ": unexpected type or shape " + shape_text(t->shape));
        if (!m) continue;
        BRASA_TRY(brasa_stage_upload(m, staging->ptr, *file, *t));
        interleave_rows_kernel<<<(unsigned)(((uint64_t)rows * out->ld + 255) / 256), 256, 0, m->ctx->stream>>>((const uint16_t *)staging->ptr, (uint16_t *)p, rows, cols, out->ld, (uint32_t)i);
        BRASA_TRY(brasa_post_launch(cmd, "interleave_rows"));
    }
    return BRASA_OK;
}

int32_t Builder::vector(const std::string &name, uint64_t n, const float **out) {
    const brasa::TensorInfo *t = file->tensor(name);
    if (!t) return fail("missing tensor " + name);
    if (t->dtype != "bf16" || t->numel() != n) return fail(name + ": unexpected type or shape " + shape_text(t->shape));
    void *p;
    BRASA_TRY(get(WEIGHTS, n * 4, &p));
    *out = (const float *)p;
    if (!m) return BRASA_OK;
    BRASA_TRY(brasa_stage_upload(m, staging->ptr, *file, *t));
    widen_bf16_kernel<<<(unsigned)((n + 255) / 256), 256, 0, m->ctx->stream>>>((const uint16_t *)staging->ptr, (float *)p, n);
    return brasa_post_launch(cmd, "widen_bf16");
}

int32_t Builder::rope(double base, uint32_t dims, const float **cos_t, const float **sin_t) {
    for (const Table &t : tables_)
        if (t.base == base && t.dims == dims) {
            *cos_t = t.c;
            *sin_t = t.s;
            return BRASA_OK;
        }
    const size_t n = (size_t)limits.ctx * dims / 2;
    void *c, *s;
    BRASA_TRY(get(WORKSPACE, n * 4, &c));
    BRASA_TRY(get(WORKSPACE, n * 4, &s));
    if (m) {
        std::vector<float> hc(n), hs(n);
        BRASA_TRY(brasa_rope_table(base, dims, limits.ctx, hc.data(), hs.data()));
        BRASA_CUDA(m->ctx, cudaMemcpyAsync(c, hc.data(), n * 4, cudaMemcpyHostToDevice, m->ctx->stream));
        BRASA_CUDA(m->ctx, cudaMemcpyAsync(s, hs.data(), n * 4, cudaMemcpyHostToDevice, m->ctx->stream));
        BRASA_CUDA(m->ctx, cudaStreamSynchronize(m->ctx->stream));
    }
    tables_.push_back(Table{base, dims, (const float *)c, (const float *)s});
    *cos_t = (const float *)c;
    *sin_t = (const float *)s;
    return BRASA_OK;
}

// ---- the model ---------------------------------------------------------------------------------------------------------

// mixers by the name their configuration entries carry
std::unique_ptr<Mixer> make_mixer(const std::string &type) {
    if (type == "latent_attention") return make_latent_attention();
    if (type == "channel_delta") return make_channel_delta();
    if (type == "delta") return make_delta();
    if (type == "parallel") return make_parallel();
    return nullptr;
}

StackModel::StackModel(const std::string &family) : wiring(family == "Gugedra" ? Wiring::SANDWICH : Wiring::BRANCHES) {}

bool StackModel::configure(const brasa::Json &c, std::string &err) {
    const brasa::Json *norm = c.get("norm"), *ls = c.get("layers");
    if (!norm || !ls || ls->kind != brasa::Json::Arr || ls->arr.empty()) return err = "config.json: norm or layers is missing", false;
    double e, v;
    if (!read_u32(c, "vocab", &vocab, err) || !read_u32(c, "width", &width, err) || !read_f64(*norm, "eps", &e, err)) return false;
    eps = (float)e;
    if (wiring == Wiring::BRANCHES) {
        const brasa::Json *emb = c.get("embedding");
        if (!emb) return err = "config.json: embedding is missing", false;
        if (!read_f64(*emb, "scale", &v, err)) return false;
        embed_scale = (float)v;
        if (!read_f64(c, "logit_scale", &v, err)) return false;
        logit_scale = (float)v;
    } else {
        const brasa::Json *side = c.get("token_side");
        if (side && side->kind == brasa::Json::Obj && !read_u32(*side, "dim", &side_dim, err)) return false;
        if (!read_f64(c, "logit_softcap", &v, err)) return false;
        if (!(v > 0.0)) return err = "config.json: logit_softcap must be positive", false;
        logit_cap = (float)v;
    }
    for (const brasa::Json &j : ls->arr) {
        layers.emplace_back();
        StackLayer &l = layers.back();
        const brasa::Json *type = j.get("type"), *mix = j.get("mixer"), *mlp = j.get("mlp");
        if (!type || type->kind != brasa::Json::Str || !mix || mix->kind != brasa::Json::Obj) return err = "config.json: a layer without type or mixer", false;
        l.mixer = make_mixer(type->str);
        if (!l.mixer) return err = "config.json: unknown mixer " + type->str, false;
        if (!l.mixer->configure(*mix, width, eps, err)) return false;
        if (mlp && mlp->kind == brasa::Json::Obj) {
            const brasa::Json *kind = mlp->get("kind");
            if (!kind || kind->kind != brasa::Json::Str || kind->str != "dense") return err = "config.json: unknown feed-forward kind", false;
            if (!read_u32(*mlp, "ff", &l.ff, err)) return false;
        }
    }
    return true;
}

int32_t StackModel::build(Builder &b) {
    const bool sandwich = wiring == Wiring::SANDWICH;
    f32 = b.f32;
    BRASA_TRY(b.matrix("embed", vocab, width, &embed));
    if (side_dim) BRASA_TRY(b.matrix("side.embed", vocab, (uint32_t)layers.size() * side_dim, &side_embed));
    uint32_t widest_out[2] = {8, 8}, widest_ff = 8;
    auto norm = [&](const std::string &name, const float **w, const float **bias) {
        BRASA_TRY(b.vector(name, width, w));
        return sandwich ? BRASA_OK : b.vector(name + ".b", width, bias);
    };
    for (size_t i = 0; i < layers.size(); ++i) {
        StackLayer &l = layers[i];
        const std::string p = "l" + std::to_string(i) + ".";
        BRASA_TRY(norm(p + "norm1", &l.norm_w[0], &l.norm_b[0]));
        if (sandwich) BRASA_TRY(b.vector(p + "norm1b", width, &l.post_w[0]));
        BRASA_TRY(l.mixer->build(b, p + "mix."));
        if (l.mixer->outs.empty() || l.mixer->outs.size() > 2 || (!sandwich && l.mixer->outs.size() > 1)) return b.fail(p + "mix: a mixer this wiring has no place for");
        for (size_t k = 0; k < l.mixer->outs.size(); ++k) widest_out[k] = std::max(widest_out[k], up8(l.mixer->outs[k].cols));
        if (side_dim) {
            BRASA_TRY(b.matrix(p + "side.gate", side_dim, width, &l.side_gate));
            BRASA_TRY(b.matrix(p + "side.proj", width, side_dim, &l.side_proj));
            BRASA_TRY(b.vector(p + "side.norm", width, &l.side_w));
        }
        if (!l.ff) continue;
        BRASA_TRY(norm(p + "norm2", &l.norm_w[1], &l.norm_b[1]));
        BRASA_TRY(b.matrix(p + "mlp.down", width, l.ff, &l.down));
        if (sandwich) {
            BRASA_TRY(b.vector(p + "norm2b", width, &l.post_w[1]));
            BRASA_TRY(b.interleaved(p + "mlp.gate", p + "mlp.up", l.ff, width, &l.up));
        } else {
            BRASA_TRY(b.matrix(p + "mlp.up", l.ff, width, &l.up));
            BRASA_TRY(b.vector(p + "mlp.up.b", l.ff, &l.up_b));
            BRASA_TRY(b.vector(p + "mlp.down.b", width, &l.down_b));
        }
        widest_ff = std::max(widest_ff, (l.ff + 31) / 32 * 32);
    }
    BRASA_TRY(norm("final.norm", &final_w, &final_b));
    BRASA_TRY(b.matrix("head", vocab, width, &head));
    const uint64_t t = b.limits.max_tokens, e = b.elem();
    uint64_t scratch_n = 0;
    for (StackLayer &l : layers) scratch_n = std::max(scratch_n, l.mixer->scratch_bytes());
    auto ws = [&](uint64_t n, void **out) { return b.get(Builder::WORKSPACE, n, out); };
    BRASA_TRY(ws(t * width * 4, (void **)&x));
    for (int i = 0; i < (sandwich ? 1 : 2); ++i) BRASA_TRY(ws(t * up8(width) * e, &h[i]));
    for (int i = 0; i < (sandwich ? 2 : 1); ++i) BRASA_TRY(ws(std::max(t * e, (uint64_t)4) * widest_out[i], &mixed[i]));  // (one token's vectors are f32 in every mode)
    BRASA_TRY(ws(std::max(t * e, (uint64_t)8) * widest_ff, &act));  // (one token: gate and up values)
    if (sandwich) {
        BRASA_TRY(ws(t * width * 4, (void **)&y));
        BRASA_TRY(ws((uint64_t)width * 4, (void **)&x2));
        BRASA_TRY(ws(std::max(t * e, (uint64_t)4) * up8(side_dim ? side_dim : 8), &side));
    }
    BRASA_TRY(ws(scratch_n, (void **)&scratch));
    BRASA_TRY(ws((uint64_t)b.limits.max_logit_rows * up8(width) * e, &head_in));
    BRASA_TRY(ws((uint64_t)b.limits.max_logit_rows * 4, (void **)&row_ids));
    return BRASA_OK;
}

int32_t StackModel::layers_run(brasa_cmd *cmd, size_t l0, size_t l1, uint32_t tokens, uint32_t pos0) {
    if (wiring == Wiring::SANDWICH && l0 < l1)
        BRASA_TRY(brasa_add_rms_norm_launch(cmd, x, nullptr, nullptr, nullptr, layers[l0].norm_w[0], h[0], nullptr, tokens, width, up8(width), eps, f32));
    for (size_t i = l0; i < l1; ++i)
        BRASA_TRY(wiring == Wiring::SANDWICH ? sandwich_run(cmd, i, tokens, pos0, i + 1 < l1 ? layers[i + 1].norm_w[0] : nullptr) : branches_run(cmd, i, tokens, pos0));
    return BRASA_OK;
}

int32_t StackModel::layers_step(brasa_cmd *cmd, size_t l0, size_t l1, const uint32_t *dev_pos, Pending &p) {
    p = Pending{x, nullptr, nullptr};
    for (size_t i = l0; i < l1; ++i) BRASA_TRY(wiring == Wiring::SANDWICH ? sandwich_step(cmd, i, dev_pos, p) : branches_step(cmd, i, dev_pos));
    return BRASA_OK;
}

int32_t StackModel::settle(brasa_cmd *cmd, const Pending &p) {
    if (!p.y) return BRASA_OK;
    return brasa_add_rms_norm_launch(cmd, p.x, p.y, p.wy, x, nullptr, nullptr, nullptr, 1, width, up8(width), eps, true);
}

Run StackModel::run_of(brasa_cmd *cmd, size_t li, uint32_t tokens, uint32_t pos0, const uint32_t *dev_pos) {
    const std::vector<MixerOut> &o = layers[li].mixer->outs;
    Run r{cmd, tokens, pos0, dev_pos, f32, dev_pos ? nullptr : h[0], dev_pos ? 0u : up8(width), {mixed[0], mixed[1]}, {up8(o[0].cols), o.size() > 1 ? up8(o[1].cols) : 0u}, scratch};
    return r;
}

// the mixer's projections, and another product on the way
int32_t StackModel::project_run(const Run &r, size_t li, const LinearProblem *more) {
    std::vector<GemvProblem> g;
    layers[li].mixer->project(r, g);
    std::vector<LinearProblem> p;
    for (const GemvProblem &q : g) p.push_back(q.p);
    if (more) p.push_back(*more);
    return brasa_linear_launch(r.cmd, p.data(), (uint32_t)p.size(), f32);
}

// The vectors of one token ahead of the mixer's output projections.
GemvInput StackModel::mixed_input(const StackLayer &l) const {
    GemvInput in;
    in.eps = eps;
    for (size_t k = 0; k < l.mixer->outs.size(); ++k) {
        const MixerOut &o = l.mixer->outs[k];
        in.v[k] = (const float *)mixed[k];
        in.len[k] = o.cols;
        in.parts[k] = o.parts;
        in.vw[k] = o.part_w;
        in.vscale[k] = o.part_scale;
    }
    return in;
}

// ---- Wiring::BRANCHES ----------------------------------------------------------------------------------------------------
int32_t StackModel::branches_run(brasa_cmd *cmd, size_t li, uint32_t tokens, uint32_t pos0) {
    StackLayer &l = layers[li];
    const uint32_t ldh = up8(width);
    BRASA_TRY(brasa_layer_norm_launch(cmd, x, nullptr, tokens, width, eps, l.norm_w, l.norm_b, h, l.ff ? 2 : 1, ldh, f32));
    const Run r = run_of(cmd, li, tokens, pos0, nullptr);
    LinearProblem u;
    u.seg[0] = segment(l.up, h[1], ldh);
    u.rows = l.ff;
    u.tokens = tokens;
    u.y = act;
    u.ldy = up8(l.ff);
    u.y_bf16 = !f32;
    u.bias = l.up_b;
    u.act = LINEAR_ACT_RELU2;
    BRASA_TRY(project_run(r, li, l.ff ? &u : nullptr));
    BRASA_TRY(l.mixer->mix(r));
    LinearProblem o;
    o.seg[0] = segment(l.mixer->outs[0], mixed[0], r.ldo[0]);
    if (l.ff) o.seg[1] = segment(l.down, act, up8(l.ff));
    o.rows = width;
    o.tokens = tokens;
    o.y = x;
    o.ldy = width;
    o.bias = l.down_b;
    o.resid = x;
    return brasa_linear_launch(cmd, &o, 1, f32);
}

// The same for one token whose position the device holds.
int32_t StackModel::branches_step(brasa_cmd *cmd, size_t li, const uint32_t *dev_pos) {
    StackLayer &l = layers[li];
    const Run r = run_of(cmd, li, 1, 0, dev_pos);
    std::vector<GemvProblem> p;
    l.mixer->project(r, p);
    GemvInput in;
    in.x = x;
    in.width = width;
    in.eps = eps;
    for (int i = 0; i < (l.ff ? 2 : 1); ++i) {
        in.w[i] = l.norm_w[i];
        in.b[i] = l.norm_b[i];
    }
    if (l.ff) {
        GemvProblem u;
        u.p.seg[0] = segment(l.up, nullptr, 0);
        u.input[0] = 1;
        u.p.rows = l.ff;
        u.p.y = act;
        u.p.bias = l.up_b;
        u.p.act = LINEAR_ACT_RELU2;
        p.push_back(u);
    }
    BRASA_TRY(brasa_linear_gemv_launch(cmd, in, p.data(), (uint32_t)p.size()));
    BRASA_TRY(l.mixer->mix(r));
    GemvInput oin = mixed_input(l);
    GemvProblem o;
    o.p.seg[0] = segment(l.mixer->outs[0], nullptr, 0);
    if (l.ff) {
        oin.v[1] = (const float *)act;
        oin.len[1] = l.ff;
        o.p.seg[1] = segment(l.down, nullptr, 0);
    }
    o.p.rows = width;
    o.p.y = x;
    o.p.bias = l.down_b;
    o.p.resid = x;
    return brasa_linear_gemv_launch(cmd, oin, &o, 1);
}

// ---- Wiring::SANDWICH ----------------------------------------------------------------------------------------------------
// side.gate's product with the residual stream, times the layer's part of the tokens' second embedding
LinearProblem StackModel::side_gate_problem(size_t li) const {
    LinearProblem g;
    g.seg[0] = segment(layers[li].side_gate, h[0], up8(width));
    g.rows = side_dim;
    g.y = side;
    g.ldy = up8(side_dim);
    g.act = LINEAR_ACT_GELU_TANH;
    g.mul = side_embed.p + li * side_dim;
    g.ldm = side_embed.ld;
    g.mul_ids = ids;
    return g;
}

// A layer whose normed input is in h[0]; leaves x, and x normed with next_w (if given) in h[0].
int32_t StackModel::sandwich_run(brasa_cmd *cmd, size_t li, uint32_t tokens, uint32_t pos0, const float *next_w) {
    StackLayer &l = layers[li];
    const uint32_t ldh = up8(width);
    const Run r = run_of(cmd, li, tokens, pos0, nullptr);
    // x += y / rms(y) * wy; the next input to h[0]
    auto add = [&](const float *wy, const float *w, bool input) {
        return brasa_add_rms_norm_launch(cmd, x, y, wy, x, w, input ? h[0] : nullptr, nullptr, tokens, width, ldh, eps, f32);
    };
    auto result = [&](LinearProblem p) {
        p.rows = width;
        p.tokens = tokens;
        p.y = y;
        p.ldy = width;
        return brasa_linear_launch(cmd, &p, 1, f32);
    };
    BRASA_TRY(project_run(r, li, nullptr));
    BRASA_TRY(l.mixer->mix(r));
    LinearProblem o;
    for (size_t k = 0; k < l.mixer->outs.size(); ++k) o.seg[k] = segment(l.mixer->outs[k], mixed[k], r.ldo[k]);
    BRASA_TRY(result(o));
    if (l.ff) {
        BRASA_TRY(add(l.post_w[0], l.norm_w[1], true));
        LinearProblem u;
        u.seg[0] = segment(l.up, h[0], ldh);
        u.rows = l.up.rows;
        u.tokens = tokens;
        u.y = act;
        u.ldy = l.up.rows / 2;
        u.y_bf16 = !f32;
        u.act = LINEAR_ACT_SWIGLU;
        BRASA_TRY(brasa_linear_launch(cmd, &u, 1, f32));
        LinearProblem d;
        d.seg[0] = segment(l.down, act, l.up.rows / 2);
        BRASA_TRY(result(d));
    }
    const float *wy = l.post_w[l.ff ? 1 : 0];
    if (!side_dim) return add(wy, next_w, next_w != nullptr);
    BRASA_TRY(add(wy, nullptr, true));
    LinearProblem g = side_gate_problem(li);
    g.tokens = tokens;
    g.y_bf16 = !f32;
    BRASA_TRY(brasa_linear_launch(cmd, &g, 1, f32));
    LinearProblem s;
    s.seg[0] = segment(l.side_proj, side, up8(side_dim));
    BRASA_TRY(result(s));
    return add(l.side_w, next_w, next_w != nullptr);
}

// x with what is pending as a product's input; afterwards nothing is pending.
GemvInput StackModel::pending_input(Pending &p, GemvNorm norm, const float *w) {
    GemvInput in;
    in.x = p.x;
    in.norm = norm;
    in.width = width;
    in.eps = eps;
    in.w[0] = w;
    if (p.y) {
        in.y = p.y;
        in.wy = p.wy;
        in.x_out = p.x == x ? x2 : x;
        p = Pending{in.x_out, nullptr, nullptr};
    }
    return in;
}

int32_t StackModel::sandwich_step(brasa_cmd *cmd, size_t li, const uint32_t *dev_pos, Pending &p) {
    StackLayer &l = layers[li];
    const Run r = run_of(cmd, li, 1, 0, dev_pos);
    auto result = [&](const GemvInput &in, GemvProblem q, const float *wy) {
        q.p.rows = width;
        q.p.y = y;
        p.y = y;
        p.wy = wy;
        return brasa_linear_gemv_launch(cmd, in, &q, 1);
    };
    std::vector<GemvProblem> g;
    l.mixer->project(r, g);
    BRASA_TRY(brasa_linear_gemv_launch(cmd, pending_input(p, GEMV_RMS_NORM, l.norm_w[0]), g.data(), (uint32_t)g.size()));
    BRASA_TRY(l.mixer->mix(r));
    GemvProblem o;
    for (size_t k = 0; k < l.mixer->outs.size(); ++k) o.p.seg[k] = segment(l.mixer->outs[k], nullptr, 0);
    BRASA_TRY(result(mixed_input(l), o, l.post_w[0]));
    if (l.ff) {
        GemvProblem u;
        u.p.seg[0] = segment(l.up, nullptr, 0);
        u.p.rows = l.up.rows;
        u.p.y = act;
        BRASA_TRY(brasa_linear_gemv_launch(cmd, pending_input(p, GEMV_RMS_NORM, l.norm_w[1]), &u, 1));
        GemvInput in;
        in.v[0] = (const float *)act;
        in.len[0] = l.ff;
        in.gated = true;
        GemvProblem d;
        d.p.seg[0] = segment(l.down, nullptr, 0);
        BRASA_TRY(result(in, d, l.post_w[1]));
    }
    if (!side_dim) return BRASA_OK;
    GemvProblem sg;
    sg.p = side_gate_problem(li);
    BRASA_TRY(brasa_linear_gemv_launch(cmd, pending_input(p, GEMV_PLAIN, nullptr), &sg, 1));
    GemvInput in;
    in.v[0] = (const float *)side;
    in.len[0] = side_dim;
    GemvProblem sp;
    sp.p.seg[0] = segment(l.side_proj, nullptr, 0);
    return result(in, sp, l.side_w);
}

// ---- logits --------------------------------------------------------------------------------------------------------------
// rows: places among the run's tokens (device array) whose logits go to `logits`, in order
int32_t StackModel::logits_of(brasa_cmd *cmd, const uint32_t *rows, uint32_t n, float *logits) {
    if (wiring == Wiring::SANDWICH) {
        BRASA_TRY(brasa_add_rms_norm_launch(cmd, x, nullptr, nullptr, nullptr, final_w, head_in, rows, n, width, up8(width), eps, f32));
    } else {
        const float *w[2] = {final_w, nullptr}, *b[2] = {final_b, nullptr};
        void *out[2] = {head_in, nullptr};
        BRASA_TRY(brasa_layer_norm_launch(cmd, x, rows, n, width, eps, w, b, out, 1, up8(width), f32));
    }
    LinearProblem p;
    p.seg[0] = segment(head, head_in, up8(width));
    p.rows = vocab;
    p.tokens = n;
    p.y = logits;
    p.ldy = vocab;
    p.scale = logit_scale;
    p.cap = logit_cap;
    return brasa_linear_launch(cmd, &p, 1, f32);
}

int32_t StackModel::logits_step(brasa_cmd *cmd, const Pending &pending, float *logits) {
    Pending q = pending;
    GemvInput in;
    if (wiring == Wiring::SANDWICH) {
        in = pending_input(q, GEMV_RMS_NORM, final_w);
        in.x_out = nullptr;
    } else {
        in.x = x;
        in.width = width;
        in.eps = eps;
        in.w[0] = final_w;
        in.b[0] = final_b;
    }
    GemvProblem p;
    p.p.seg[0] = segment(head, nullptr, 0);
    p.p.rows = vocab;
    p.p.y = logits;
    p.p.scale = logit_scale;
    p.p.cap = logit_cap;
    return brasa_linear_gemv_launch(cmd, in, &p, 1);
}

// ---- the families --------------------------------------------------------------------------------------------------------
namespace {

bool describe(const brasa::WeightFile &f, brasa_model_shape *shape, brasa_config *cfg, std::string &err) {
    StackModel s(f.family());
    if (!s.configure(f.config(), err)) return false;
    if (cfg) {
        *cfg = brasa_config{};
        cfg->hidden = s.width;
        cfg->layers = (uint32_t)s.layers.size();
        cfg->vocab = cfg->head_rows = s.vocab;
        cfg->max_position = 0x7fffffff;
        cfg->eps = s.eps;
    }
    if (shape) {
        Builder b;
        b.file = &f;
        b.limits = brasa_limits{1, 1, 1, BRASA_KV_BF16};
        if (s.build(b) != BRASA_OK) return err = b.err, false;
        *shape = brasa_model_shape{};
        shape->weight_bytes = b.bytes[Builder::WEIGHTS];
        shape->layers = (uint32_t)s.layers.size();
        shape->hidden = s.width;
        shape->vocab = s.vocab;
    }
    return true;
}

// buffers of brasa_model_load beside the builder's
uint64_t common_workspace(const brasa_limits &l, uint32_t vocab) {
    return brasa_plan_buffer_bytes((uint64_t)l.max_tokens * 4) + brasa_plan_buffer_bytes((uint64_t)l.max_logit_rows * vocab * 4);
}

int32_t check_kv(brasa_ctx *ctx, int32_t kv) {
    BRASA_REQUIRE(ctx, kv == BRASA_KV_F32 || kv == BRASA_KV_BF16, "this family runs in bf16 or f32 (cache type %d)", kv);
    return BRASA_OK;
}

int32_t plan(brasa_ctx *ctx, const brasa::WeightFile &f, const brasa_session_shape &s, brasa_memory_plan *out) {
    BRASA_TRY(check_kv(ctx, s.kv));
    StackModel sm(f.family());
    Builder b;
    b.file = &f;
    b.limits = brasa_limits{s.ctx, std::min(s.max_tokens, s.ctx), s.max_logit_rows, s.kv};
    b.f32 = s.kv == BRASA_KV_F32;
    if (!sm.configure(f.config(), b.err) || sm.build(b) != BRASA_OK) return brasa_fail(ctx, BRASA_EIO, "%s", b.err.c_str());
    out->weights = b.bytes[Builder::WEIGHTS];
    out->kv = b.bytes[Builder::STATE];
    out->workspace = b.bytes[Builder::WORKSPACE] + common_workspace(b.limits, sm.vocab);
    out->overhead = 256ull << 20;
    out->total = out->weights + out->kv + out->workspace + out->overhead;
    return BRASA_OK;
}

int32_t load(brasa_model *m, const brasa::WeightFile &f, brasa_cmd *cmd, brasa_buf *staging) {
    brasa_ctx *ctx = m->ctx;
    BRASA_TRY(check_kv(ctx, m->limits.kv));
    m->stack = new StackModel(f.family());
    std::string err;
    if (!m->stack->configure(f.config(), err)) return brasa_fail(ctx, BRASA_EIO, "%s", err.c_str());
    Builder b;
    b.m = m;
    b.file = &f;
    b.cmd = cmd;
    b.staging = staging;
    b.limits = m->limits;
    b.f32 = m->limits.kv == BRASA_KV_F32;
    BRASA_TRY(m->stack->build(b));
    m->stack->reached.assign(m->cfg.layers, 0);
    m->alloc.weights = b.bytes[Builder::WEIGHTS];
    m->alloc.kv = b.bytes[Builder::STATE];
    m->alloc.workspace = b.bytes[Builder::WORKSPACE] + common_workspace(m->limits, m->cfg.vocab);
    return BRASA_OK;
}

void release(brasa_model *m) {
    delete m->stack;
    m->stack = nullptr;
}

int32_t begin(brasa_model *m, uint32_t pos0, uint32_t l0, uint32_t l1) {
    for (uint32_t i = l0; i < l1; ++i)
        BRASA_REQUIRE(m->ctx, pos0 == 0 || m->stack->reached[i] == pos0,
                      "position %u: the sequence's state stands at %u, from where it can go on or start over at 0", pos0, m->stack->reached[i]);
    // until the work is known to be queued the state counts as lost: only position 0 is open
    for (uint32_t i = l0; i < l1; ++i) m->stack->reached[i] = UINT32_MAX;
    return BRASA_OK;
}
void finish(brasa_model *m, uint32_t pos, uint32_t l0, uint32_t l1) {
    for (uint32_t i = l0; i < l1; ++i) m->stack->reached[i] = pos;
}
uint32_t reached(brasa_model *m) {
    uint32_t p = m->stack->reached[0];
    for (uint32_t q : m->stack->reached)
        if (q != p) return UINT32_MAX;
    return p;
}

int32_t embed_tokens(brasa_model *m, brasa_cmd *cmd, uint32_t tokens) {
    StackModel &s = *m->stack;
    s.ids = (const uint32_t *)m->ids->ptr;
    return brasa_embed_bf16_launch(cmd, s.embed.p, s.embed.ld, s.vocab, s.width, s.embed_scale, s.ids, s.x, tokens);
}

int32_t step_kernels(brasa_model *m, brasa_cmd *cmd) {
    StackModel &s = *m->stack;
    Pending p;
    BRASA_TRY(embed_tokens(m, cmd, 1));
    BRASA_TRY(s.layers_step(cmd, 0, s.layers.size(), (const uint32_t *)m->dev_state->ptr, p));
    BRASA_TRY(s.logits_step(cmd, p, F(m->logits)));
    return brasa_argmax_launch(cmd, F(m->logits), m->cfg.vocab, (uint32_t *)m->next_id->ptr);
}

int32_t forward(brasa_model *m, brasa_cmd *cmd, uint32_t tokens, uint32_t pos0, const uint32_t *rows, uint32_t n_rows) {
    StackModel &s = *m->stack;
    BRASA_TRY(embed_tokens(m, cmd, tokens));
    BRASA_TRY(s.layers_run(cmd, 0, s.layers.size(), tokens, pos0));
    if (n_rows == 0) return BRASA_OK;
    BRASA_CUDA(m->ctx, cudaMemcpyAsync(s.row_ids, rows, (size_t)n_rows * 4, cudaMemcpyHostToDevice, m->ctx->stream));
    return s.logits_of(cmd, s.row_ids, n_rows, F(m->logits));
}

int32_t run_layers(brasa_model *m, brasa_cmd *cmd, const uint32_t *ids, const float *x, float *y, uint32_t tokens, uint32_t pos0, uint32_t l0, uint32_t l1) {
    StackModel &s = *m->stack;
    const size_t n = (size_t)tokens * s.width * 4;
    s.ids = (const uint32_t *)m->ids->ptr;
    if (ids) BRASA_CUDA(m->ctx, cudaMemcpyAsync(m->ids->ptr, ids, (size_t)tokens * 4, cudaMemcpyHostToDevice, m->ctx->stream));
    BRASA_CUDA(m->ctx, cudaMemcpyAsync(s.x, x, n, cudaMemcpyHostToDevice, m->ctx->stream));
    if (tokens == 1) {
        Pending p;
        BRASA_CUDA(m->ctx, cudaMemcpyAsync(m->dev_state->ptr, &pos0, 4, cudaMemcpyHostToDevice, m->ctx->stream));
        BRASA_TRY(s.layers_step(cmd, l0, l1, (const uint32_t *)m->dev_state->ptr, p));
        BRASA_TRY(s.settle(cmd, p));
    } else {
        BRASA_TRY(s.layers_run(cmd, l0, l1, tokens, pos0));
    }
    BRASA_CUDA(m->ctx, cudaMemcpyAsync(y, s.x, n, cudaMemcpyDeviceToHost, m->ctx->stream));
    return brasa_check_cuda(m->ctx, cudaStreamSynchronize(m->ctx->stream), "run_layers");
}

}  // namespace

bool layers_read_ids(const brasa_model *m) { return m->stack && m->stack->side_dim > 0; }

const brasa_family dunuzen_family = {"Dunuzen", describe, plan, load, release, forward, step_kernels, run_layers, begin, finish, reached};
const brasa_family gugedra_family = {"Gugedra", describe, plan, load, release, forward, step_kernels, run_layers, begin, finish, reached};

}  // namespace brasa_stack
