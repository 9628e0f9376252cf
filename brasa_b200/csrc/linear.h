// Grouped products with bfloat16 weights (linear.cu): up to LINEAR_MAX problems in one launch, each
//   y[t, r] = resid[t, r] + scale * act(sum_c w[r, c] x[t, c] (+ sum_c w2[r, c] x2[t, c]) + bias[r])
// with f32 accumulation. Weights and activations are row-major; leading dimensions are multiples of 8 elements.
#pragma once
#include "brasa_internal.h"

constexpr uint32_t LINEAR_MAX = 8;
enum { LINEAR_ACT_NONE = 0, LINEAR_ACT_RELU2 = 1 };  // relu(v)^2

struct LinearSeg {
    const uint16_t *w = nullptr;  // bf16 [rows][ldw]; columns past `cols` up to ldw are zeros
    uint32_t ldw = 0;
    const void *x = nullptr;      // bf16 or f32 [tokens][ldx]
    uint32_t ldx = 0, cols = 0;
};
struct LinearProblem {
    LinearSeg seg[2];  // the second one is optional (cols == 0): one product over the concatenation of both inputs
    uint32_t rows = 0, tokens = 0;
    void *y = nullptr;  // f32 or bf16 [tokens][ldy]
    uint32_t ldy = 0;
    bool y_bf16 = false;
    const float *bias = nullptr;   // [rows]
    const float *resid = nullptr;  // f32 [tokens][ldy]; may be y itself
    int act = LINEAR_ACT_NONE;
    float scale = 1.0f;
};

// Many tokens. x_f32: the inputs are f32 and products run in f32 FMA; otherwise they are bf16 and go to tcgen05.
int32_t brasa_linear_launch(brasa_cmd *cmd, const LinearProblem *p, uint32_t n, bool x_f32);

// One token (vectors in f32; y f32): the weights stream once through all SMs. The input of every problem is a slice of the
// block's input vector, which the kernel forms itself: either one or two affine forms of the layer norm of ln.x, or a copy
// of up to two vectors one behind the other. The kernel is a programmatic dependent of the kernel before it.
struct GemvInput {
    const float *ln_x = nullptr;  // layer norm of this vector ..
    uint32_t width = 0;
    float eps = 0.0f;
    const float *w[2] = {nullptr, nullptr}, *b[2] = {nullptr, nullptr};  // .. times w[i] plus b[i]: input i
    const float *v[2] = {nullptr, nullptr};                             // or: input i = v[i], len[i] values
    uint32_t len[2] = {0, 0};
};
struct GemvProblem {
    LinearProblem p;         // tokens, ldy and the segments' x are unused
    uint32_t input[2] = {0, 1};  // which input each segment reads
};
int32_t brasa_linear_gemv_launch(brasa_cmd *cmd, const GemvInput &in, const GemvProblem *p, uint32_t n);
