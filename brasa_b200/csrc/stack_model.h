// A layer-stack model on the device (stack.cu).
#pragma once
#include "stack.h"

namespace brasa_stack {

// How a layer's sublayers hang on the residual stream x.
enum class Wiring {
    BRANCHES,  // x + mixer(norm1 x) + ff(norm2 x), layer norms, ff = down relu(up h)^2 with biases
    SANDWICH,  // x += norm1b(mixer(norm1 x)); x += norm2b(ff(norm2 x)), RMS norms, ff = down (silu(gate h) * up h); then, where the
               // configuration has "token_side", x += norm(proj (gelu(gate x) * e)), e the layer's part of the token's second embedding
};

struct StackLayer {
    std::unique_ptr<Mixer> mixer;
    const float *norm_w[2] = {nullptr, nullptr}, *norm_b[2] = {nullptr, nullptr};  // of the mixer's input, of the feed-forward's
    const float *post_w[2] = {nullptr, nullptr};                                  // SANDWICH: of their results
    uint32_t ff = 0;  // 0: no feed-forward
    Weight up, down;  // SANDWICH: up holds gate and up rows in alternating blocks of 32
    const float *up_b = nullptr, *down_b = nullptr;
    Weight side_gate, side_proj;
    const float *side_w = nullptr;
};

// SANDWICH, one token: the residual stream and a sublayer's result whose norm and addition the next product does on the way in.
struct Pending {
    const float *x = nullptr, *y = nullptr, *wy = nullptr;
};

struct StackModel {
    explicit StackModel(const std::string &family);
    Wiring wiring = Wiring::BRANCHES;
    uint32_t vocab = 0, width = 0, side_dim = 0;
    float eps = 0.0f, embed_scale = 1.0f, logit_scale = 1.0f, logit_cap = 0.0f;
    bool f32 = false;
    std::vector<StackLayer> layers;
    Weight embed, head, side_embed;
    const float *final_w = nullptr, *final_b = nullptr;
    // workspace: residual stream f32 [max_tokens][width], normed inputs, mixer outputs, feed-forward activations; SANDWICH: a
    // sublayer's result f32 [max_tokens][width], the token side's activations, a second residual stream of one token
    float *x = nullptr, *y = nullptr, *x2 = nullptr;
    void *h[2] = {nullptr, nullptr}, *mixed[2] = {nullptr, nullptr}, *act = nullptr, *side = nullptr, *head_in = nullptr;
    uint8_t *scratch = nullptr;
    uint32_t *row_ids = nullptr;
    const uint32_t *ids = nullptr;  // the run's token ids on the device (not owned)
    std::vector<uint32_t> reached;  // per layer: positions its state holds; UINT32_MAX: lost

    bool configure(const brasa::Json &c, std::string &err);
    int32_t build(Builder &b);
    // layers [l0, l1) over a run of tokens whose residual stream is x, or over one token whose position the device holds
    int32_t layers_run(brasa_cmd *cmd, size_t l0, size_t l1, uint32_t tokens, uint32_t pos0);
    int32_t layers_step(brasa_cmd *cmd, size_t l0, size_t l1, const uint32_t *dev_pos, Pending &p);
    int32_t settle(brasa_cmd *cmd, const Pending &p);  // one token: x takes what is pending
    int32_t logits_of(brasa_cmd *cmd, const uint32_t *rows, uint32_t n, float *logits);
    int32_t logits_step(brasa_cmd *cmd, const Pending &p, float *logits);

  private:
    Run run_of(brasa_cmd *cmd, size_t li, uint32_t tokens, uint32_t pos0, const uint32_t *dev_pos);
    int32_t project_run(const Run &r, size_t li, const LinearProblem *more);
    int32_t branches_run(brasa_cmd *cmd, size_t li, uint32_t tokens, uint32_t pos0);
    int32_t branches_step(brasa_cmd *cmd, size_t li, const uint32_t *dev_pos);
    int32_t sandwich_run(brasa_cmd *cmd, size_t li, uint32_t tokens, uint32_t pos0, const float *next_w);
    int32_t sandwich_step(brasa_cmd *cmd, size_t li, const uint32_t *dev_pos, Pending &p);
    GemvInput pending_input(Pending &p, GemvNorm norm, const float *w);
    GemvInput mixed_input(const StackLayer &l) const;
    LinearProblem side_gate_problem(size_t li) const;
};

}  // namespace brasa_stack
