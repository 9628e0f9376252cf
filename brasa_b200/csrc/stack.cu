// Layer-stack models (stack.h): the configuration reader, weights, workspace, the layer loop for runs of tokens and for one
// token, and the families built on it.
//
// Dunuzen: a layer adds its mixer's and its feed-forward's result to the residual stream, each computed from the same x behind
// a layer norm of its own; the feed-forward is two biased products with a squared relu between them. Both branches read the same x, so one pass over x forms both norms, the mixer's projections and
// the feed-forward's first product go into one launch, and the output projection and the feed-forward's second product are
// one product over the concatenation of their inputs that adds to x in its epilogue.
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
static std::unique_ptr<Mixer> make_mixer(const std::string &type) {
    if (type == "latent_attention") return make_latent_attention();
    if (type == "channel_delta") return make_channel_delta();
    return nullptr;
}

bool StackModel::configure(const brasa::Json &c, std::string &err) {
    const brasa::Json *norm = c.get("norm"), *emb = c.get("embedding"), *ls = c.get("layers");
    if (!norm || !emb || !ls || ls->kind != brasa::Json::Arr || ls->arr.empty()) return err = "config.json: norm, embedding or layers is missing", false;
    double e, es, lsc;
    if (!read_u32(c, "vocab", &vocab, err) || !read_u32(c, "width", &width, err) || !read_f64(*norm, "eps", &e, err) || !read_f64(*emb, "scale", &es, err) ||
        !read_f64(c, "logit_scale", &lsc, err))
        return false;
    eps = (float)e;
    embed_scale = (float)es;
    logit_scale = (float)lsc;
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
    f32 = b.f32;
    BRASA_TRY(b.matrix("embed", vocab, width, &embed));
    uint32_t widest_out = 8, widest_ff = 8;
    for (size_t i = 0; i < layers.size(); ++i) {
        StackLayer &l = layers[i];
        const std::string p = "l" + std::to_string(i) + ".";
        BRASA_TRY(b.vector(p + "norm1", width, &l.norm_w[0]));
        BRASA_TRY(b.vector(p + "norm1.b", width, &l.norm_b[0]));
        BRASA_TRY(l.mixer->build(b, p + "mix."));
        widest_out = std::max(widest_out, up8(l.mixer->out_width));
        if (!l.ff) continue;
        BRASA_TRY(b.vector(p + "norm2", width, &l.norm_w[1]));
        BRASA_TRY(b.vector(p + "norm2.b", width, &l.norm_b[1]));
        BRASA_TRY(b.matrix(p + "mlp.up", l.ff, width, &l.up));
        BRASA_TRY(b.vector(p + "mlp.up.b", l.ff, &l.up_b));
        BRASA_TRY(b.matrix(p + "mlp.down", width, l.ff, &l.down));
        BRASA_TRY(b.vector(p + "mlp.down.b", width, &l.down_b));
        widest_ff = std::max(widest_ff, up8(l.ff));
    }
    BRASA_TRY(b.vector("final.norm", width, &final_w));
    BRASA_TRY(b.vector("final.norm.b", width, &final_b));
    BRASA_TRY(b.matrix("head", vocab, width, &head));
    const uint64_t t = b.limits.max_tokens, e = b.elem();
    uint64_t scratch_n = 0;
    for (StackLayer &l : layers) scratch_n = std::max(scratch_n, l.mixer->scratch_bytes(b));
    auto ws = [&](uint64_t n, void **out) { return b.get(Builder::WORKSPACE, n, out); };
    BRASA_TRY(ws(t * width * 4, (void **)&x));
    for (int i = 0; i < 2; ++i) BRASA_TRY(ws(t * up8(width) * e, &h[i]));
    BRASA_TRY(ws(std::max(t * e, (uint64_t)4) * widest_out, &mixed));  // (one token's vectors are f32 in every mode)
    BRASA_TRY(ws(std::max(t * e, (uint64_t)4) * widest_ff, &act));
    BRASA_TRY(ws(scratch_n, (void **)&scratch));
    BRASA_TRY(ws((uint64_t)b.limits.max_logit_rows * up8(width) * e, &head_in));
    BRASA_TRY(ws((uint64_t)b.limits.max_logit_rows * 4, (void **)&row_ids));
    return BRASA_OK;
}

int32_t StackModel::layer_run(brasa_cmd *cmd, size_t li, uint32_t tokens, uint32_t pos0) {
    StackLayer &l = layers[li];
    const uint32_t ldh = up8(width);
    BRASA_TRY(brasa_layer_norm_launch(cmd, x, nullptr, tokens, width, eps, l.norm_w, l.norm_b, h, l.ff ? 2 : 1, ldh, f32));
    Run r{cmd, tokens, pos0, nullptr, f32, h[0], ldh, mixed, up8(l.mixer->out_width), scratch};
    std::vector<GemvProblem> g;
    l.mixer->project(r, g);
    std::vector<LinearProblem> p;
    for (const GemvProblem &q : g) p.push_back(q.p);
    if (l.ff) {
        LinearProblem u;
        u.seg[0] = segment(l.up, h[1], ldh);
        u.rows = l.ff;
        u.tokens = tokens;
        u.y = act;
        u.ldy = up8(l.ff);
        u.y_bf16 = !f32;
        u.bias = l.up_b;
        u.act = LINEAR_ACT_RELU2;
        p.push_back(u);
    }
    BRASA_TRY(brasa_linear_launch(cmd, p.data(), (uint32_t)p.size(), f32));
    BRASA_TRY(l.mixer->mix(r));
    LinearProblem o;
    o.seg[0] = segment(l.mixer->wo, mixed, r.ldo);
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
int32_t StackModel::layer_step(brasa_cmd *cmd, size_t li, const uint32_t *dev_pos) {
    StackLayer &l = layers[li];
    Run r{cmd, 1, 0, dev_pos, f32, nullptr, 0, mixed, up8(l.mixer->out_width), scratch};
    std::vector<GemvProblem> p;
    l.mixer->project(r, p);
    GemvInput in;
    in.ln_x = x;
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
    GemvInput oin;
    oin.v[0] = (const float *)mixed;
    oin.len[0] = l.mixer->out_width;
    GemvProblem o;
    o.p.seg[0] = segment(l.mixer->wo, nullptr, 0);
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

// rows: places among the run's tokens (device array) whose logits go to `logits`, in order
int32_t StackModel::logits_of(brasa_cmd *cmd, const uint32_t *rows, uint32_t n, float *logits) {
    const float *w[2] = {final_w, nullptr}, *b[2] = {final_b, nullptr};
    void *out[2] = {head_in, nullptr};
    BRASA_TRY(brasa_layer_norm_launch(cmd, x, rows, n, width, eps, w, b, out, 1, up8(width), f32));
    LinearProblem p;
    p.seg[0] = segment(head, head_in, up8(width));
    p.rows = vocab;
    p.tokens = n;
    p.y = logits;
    p.ldy = vocab;
    p.scale = logit_scale;
    return brasa_linear_launch(cmd, &p, 1, f32);
}

int32_t StackModel::logits_step(brasa_cmd *cmd, float *logits) {
    GemvInput in;
    in.ln_x = x;
    in.width = width;
    in.eps = eps;
    in.w[0] = final_w;
    in.b[0] = final_b;
    GemvProblem p;
    p.p.seg[0] = segment(head, nullptr, 0);
    p.p.rows = vocab;
    p.p.y = logits;
    p.p.scale = logit_scale;
    return brasa_linear_gemv_launch(cmd, in, &p, 1);
}

// ---- the family ----------------------------------------------------------------------------------------------------------
namespace {

bool describe(const brasa::WeightFile &f, brasa_model_shape *shape, brasa_config *cfg, std::string &err) {
    StackModel s;
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
    StackModel sm;
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
    m->stack = new StackModel();
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

int32_t step_kernels(brasa_model *m, brasa_cmd *cmd) {
    StackModel &s = *m->stack;
    const uint32_t *pos = (const uint32_t *)m->dev_state->ptr;
    BRASA_TRY(brasa_embed_bf16_launch(cmd, s.embed.p, s.embed.ld, s.vocab, s.width, s.embed_scale, (const uint32_t *)m->ids->ptr, s.x, 1));
    for (size_t i = 0; i < s.layers.size(); ++i) BRASA_TRY(s.layer_step(cmd, i, pos));
    BRASA_TRY(s.logits_step(cmd, F(m->logits)));
    return brasa_argmax_launch(cmd, F(m->logits), m->cfg.vocab, (uint32_t *)m->next_id->ptr);
}

int32_t forward(brasa_model *m, brasa_cmd *cmd, uint32_t tokens, uint32_t pos0, const uint32_t *rows, uint32_t n_rows) {
    StackModel &s = *m->stack;
    BRASA_TRY(brasa_embed_bf16_launch(cmd, s.embed.p, s.embed.ld, s.vocab, s.width, s.embed_scale, (const uint32_t *)m->ids->ptr, s.x, tokens));
    for (size_t i = 0; i < s.layers.size(); ++i) BRASA_TRY(s.layer_run(cmd, i, tokens, pos0));
    if (n_rows == 0) return BRASA_OK;
    BRASA_CUDA(m->ctx, cudaMemcpyAsync(s.row_ids, rows, (size_t)n_rows * 4, cudaMemcpyHostToDevice, m->ctx->stream));
    return s.logits_of(cmd, s.row_ids, n_rows, F(m->logits));
}

int32_t run_layers(brasa_model *m, brasa_cmd *cmd, const float *x, float *y, uint32_t tokens, uint32_t pos0, uint32_t l0, uint32_t l1) {
    StackModel &s = *m->stack;
    const size_t n = (size_t)tokens * s.width * 4;
    BRASA_CUDA(m->ctx, cudaMemcpyAsync(s.x, x, n, cudaMemcpyHostToDevice, m->ctx->stream));
    if (tokens == 1) BRASA_CUDA(m->ctx, cudaMemcpyAsync(m->dev_state->ptr, &pos0, 4, cudaMemcpyHostToDevice, m->ctx->stream));
    for (uint32_t i = l0; i < l1; ++i)
        BRASA_TRY(tokens == 1 ? s.layer_step(cmd, i, (const uint32_t *)m->dev_state->ptr) : s.layer_run(cmd, i, tokens, pos0));
    BRASA_CUDA(m->ctx, cudaMemcpyAsync(y, s.x, n, cudaMemcpyDeviceToHost, m->ctx->stream));
    return brasa_check_cuda(m->ctx, cudaStreamSynchronize(m->ctx->stream), "run_layers");
}

}  // namespace

const brasa_family dunuzen_family = {"Dunuzen", describe, plan, load, release, forward, step_kernels, run_layers, begin, finish, reached};

}  // namespace brasa_stack
