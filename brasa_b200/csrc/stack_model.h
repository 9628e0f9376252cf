// A layer-stack model on the device (stack.cu).
#pragma once
#include "stack.h"

namespace brasa_stack {

struct StackLayer {
    std::unique_ptr<Mixer> mixer;
    const float *norm_w[2] = {nullptr, nullptr}, *norm_b[2] = {nullptr, nullptr};  // of the mixer, of the feed-forward
    uint32_t ff = 0;  // 0: no feed-forward
    Weight up, down;
    const float *up_b = nullptr, *down_b = nullptr;
};

struct StackModel {
    uint32_t vocab = 0, width = 0;
    float eps = 0.0f, embed_scale = 1.0f, logit_scale = 1.0f;
    bool f32 = false;
    std::vector<StackLayer> layers;
    Weight embed, head;
    const float *final_w = nullptr, *final_b = nullptr;
    // workspace: residual stream f32 [max_tokens][width], normed inputs, mixer output, feed-forward activations
    float *x = nullptr;
    void *h[2] = {nullptr, nullptr}, *mixed = nullptr, *act = nullptr, *head_in = nullptr;
    uint8_t *scratch = nullptr;
    uint32_t *row_ids = nullptr;
    std::vector<uint32_t> reached;  // per layer: positions its state holds; UINT32_MAX: lost

    bool configure(const brasa::Json &c, std::string &err);
    int32_t build(Builder &b);
    int32_t layer_run(brasa_cmd *cmd, size_t li, uint32_t tokens, uint32_t pos0);
    int32_t layer_step(brasa_cmd *cmd, size_t li, const uint32_t *dev_pos);
    int32_t logits_of(brasa_cmd *cmd, const uint32_t *rows, uint32_t n, float *logits);
    int32_t logits_step(brasa_cmd *cmd, float *logits);
};

}  // namespace brasa_stack
