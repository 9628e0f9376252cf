// The model's device state, shared by model.cu (single-sequence path) and batch.cu (batched serving path).
#pragma once
#include <vector>

#include "brasa_internal.h"
#include "decode_token.h"
#include "host_util.h"

bool brasa_gemm_swiglu_fuses(const brasa_qmatrix &wg, const brasa_qmatrix &wu, uint32_t tokens);

namespace brasa_model_detail {

constexpr uint32_t GEMV_MAX_TOKENS = 8;  // qwen3.rs:276

struct Matrix {
    brasa_buf *buf = nullptr;
    brasa_qmatrix q{};
};

struct Layer {
    brasa_buf *attn_norm, *q_norm, *k_norm, *ffn_norm;
    Matrix wq, wk, wv, wo, gate, up, down;
};

inline brasa_arg A(brasa_buf *b, uint64_t off = 0) { return brasa_arg{b, off}; }
inline float *F(brasa_buf *b, uint64_t off_floats = 0) { return (float *)b->ptr + off_floats; }

struct Stager;

}  // namespace brasa_model_detail

using namespace brasa_model_detail;

namespace brasa_stack {
struct StackModel;
}

// What a model family provides to the model, session and planner entry points (model.cu holds the table of families).
struct brasa_family {
    const char *name;  // `.brasa` model family, or config.json "architecture"
    bool (*describe)(const brasa::WeightFile &f, brasa_model_shape *shape, brasa_config *cfg, std::string &err);
    int32_t (*plan)(brasa_ctx *ctx, const brasa::WeightFile &f, const brasa_session_shape &s, brasa_memory_plan *out);
    // weights, per-sequence state and workspace of a model whose ctx, cfg and limits are set; staging holds the largest tensor
    int32_t (*load)(brasa_model *m, const brasa::WeightFile &f, brasa_cmd *cmd, brasa_buf *staging);
    void (*release)(brasa_model *m);
    // ids in m->ids; logits of the given places among the tokens (host array) go to m->logits
    int32_t (*forward)(brasa_model *m, brasa_cmd *cmd, uint32_t tokens, uint32_t pos0, const uint32_t *rows, uint32_t n_rows);
    // one token m->ids[0] at the position in m->dev_state[0]: logits to m->logits, the greedy choice to m->next_id
    int32_t (*step)(brasa_model *m, brasa_cmd *cmd);
    // ids: of the tokens; may be null where the layers do not read them
    int32_t (*run_layers)(brasa_model *m, brasa_cmd *cmd, const uint32_t *ids, const float *x, float *y, uint32_t tokens, uint32_t pos0, uint32_t l0, uint32_t l1);
    // Families whose state cannot be rewound: begin checks that layers [l0, l1) can take a run at pos0 (their own position, or
    // 0), finish notes the position they have reached, reached tells it. All null where any cached position can be continued from.
    int32_t (*begin)(brasa_model *m, uint32_t pos0, uint32_t l0, uint32_t l1);
    void (*finish)(brasa_model *m, uint32_t pos, uint32_t l0, uint32_t l1);
    uint32_t (*reached)(brasa_model *m);
};
namespace brasa_stack {
extern const brasa_family dunuzen_family, gugedra_family;
bool layers_read_ids(const brasa_model *m);
}
// A tensor's bytes to dst on the device, through the loading model's pinned staging buffers.
int32_t brasa_stage_upload(brasa_model *m, void *dst, const brasa::WeightFile &f, const brasa::TensorInfo &t);

struct brasa_model {
    brasa_ctx *ctx = nullptr;
    const brasa_family *family = nullptr;
    brasa_stack::StackModel *stack = nullptr;  // families built on the layer stack (stack.cu); the Qwen3 members below stay empty
    brasa_tp *tp = nullptr;  // set for a tensor-parallel shard: residual adds are sums over ranks (not owned)
    brasa_config cfg{};
    brasa_limits limits{};
    int32_t prefill_precision = BRASA_PREFILL_F16;
    Matrix embed, head;  // head aliases embed when tied
    brasa_buf *final_norm = nullptr;
    std::vector<Layer> layers;
    brasa_buf *rope_cos = nullptr, *rope_sin = nullptr;
    brasa_buf *kc = nullptr, *vc = nullptr;  // [layers, cap, kv_heads, head_dim] in the cache type
    uint32_t cap = 0;
    // workspace
    brasa_buf *x = nullptr, *h = nullptr, *q = nullptr, *k_new = nullptr, *v_new = nullptr, *attn = nullptr, *xh = nullptr,
              *gate = nullptr, *up = nullptr, *ids = nullptr, *norm_out = nullptr, *ss = nullptr, *partials = nullptr, *logits = nullptr,
              *next_id = nullptr, *out_ids = nullptr, *dev_state = nullptr;  // dev_state: u32 pos, out_count, attention counters
    brasa_graph *decode_graph = nullptr;  // one decode step: embed .. lm_head, argmax, advance
    brasa_token_program *token_prog = nullptr;  // the same step as one persistent kernel, when the shapes allow
    bool token_prog_tried = false;
    uint64_t partials_len = 0;
    brasa_allocated alloc{};
    std::vector<brasa_buf *> owned;
    uint32_t *pinned_id = nullptr;  // pinned host word for the per-step token read
    struct Stager *stager = nullptr;  // pinned staging of the file's bytes while the model loads (null afterwards)
    double load_seconds = 0.0;        // wall time of brasa_model_load, file bytes read included
    uint64_t load_bytes = 0;          // tensor bytes that went to the device
};

