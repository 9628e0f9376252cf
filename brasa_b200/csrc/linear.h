// Grouped products with bfloat16 weights (linear.cu): up to LINEAR_MAX problems in one launch, each
//   y[t, r] = resid[t, r] + mul[ids[t], r] * softcap(scale * act(sum_c w[r, c] x[t, c] (+ sum_c w2[r, c] x2[t, c]) + bias[r]))
// with f32 accumulation; bias, softcap(v) = cap tanh(v / cap), mul and resid are optional. Weights and activations are row-major;
// leading dimensions are multiples of 8 elements.
#pragma once
#include "brasa_internal.h"

constexpr uint32_t LINEAR_MAX = 8;
// RELU2: relu(v)^2. GELU_TANH: 0.5 v (1 + tanh(sqrt(2 / pi) (v + 0.044715 v^3))). SWIGLU: the rows come in alternating blocks of
// 32 gate and 32 up rows (rows a multiple of 64) and y has half as many, silu(gate) * up (no bias, scale, cap, mul or resid);
// many tokens only: the GEMV writes both kinds of rows and the product behind it forms them from there (GemvInput::gated).
enum { LINEAR_ACT_NONE = 0, LINEAR_ACT_RELU2 = 1, LINEAR_ACT_GELU_TANH = 2, LINEAR_ACT_SWIGLU = 3 };

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
    float scale = 1.0f, cap = 0.0f;  // cap 0: none
    const uint16_t *mul = nullptr;   // bf16 [..][ldm]; token t takes row mul_ids[t] (device array)
    uint32_t ldm = 0;
    const uint32_t *mul_ids = nullptr;
    uint32_t out_rows() const { return act == LINEAR_ACT_SWIGLU ? rows / 2 : rows; }
};

// Many tokens. x_f32: the inputs are f32 and products run in f32 FMA; otherwise they are bf16 and go to tcgen05.
int32_t brasa_linear_launch(brasa_cmd *cmd, const LinearProblem *p, uint32_t n, bool x_f32);

// One token (vectors in f32; y f32): the weights stream once through all SMs. The input of every problem is a slice of the
// block's input vector, which the kernel forms itself. Either from the residual stream x: one or two affine forms of its layer
// norm; or x plus y / rms(y) * wy where y is given (a sublayer's normed result; the sum also goes to x_out, which must not be
// x), as the RMS norm times w[0] or as it is. Or from up to two vectors one behind the other, each as it is, in equal
// parts over their root mean squares, or silu(gate) * up out of alternating blocks of 32. The kernel is a programmatic
// dependent of the kernel before it.
enum GemvNorm { GEMV_LAYER_NORM, GEMV_RMS_NORM, GEMV_PLAIN };
struct GemvInput {
    const float *x = nullptr;
    GemvNorm norm = GEMV_LAYER_NORM;
    uint32_t width = 0;
    float eps = 0.0f;
    const float *y = nullptr, *wy = nullptr;
    float *x_out = nullptr;
    const float *w[2] = {nullptr, nullptr}, *b[2] = {nullptr, nullptr};  // layer norm: input i = norm * w[i] + b[i]
    const float *v[2] = {nullptr, nullptr};                             // or: input i = v[i], len[i] values
    uint32_t len[2] = {0, 0};
    uint32_t parts[2] = {0, 0};  // > 0: v[i] in that many equal parts, each over its root mean square (eps), times vw[i] * vscale[i]
    const float *vw[2] = {nullptr, nullptr};
    float vscale[2] = {1.0f, 1.0f};
    bool gated = false;  // v[0]: alternating blocks of 32 gate and up values, len[0] results
};
struct GemvProblem {
    LinearProblem p;         // tokens, ldy and the segments' x are unused
    uint32_t input[2] = {0, 1};  // which input each segment reads
};
int32_t brasa_linear_gemv_launch(brasa_cmd *cmd, const GemvInput &in, const GemvProblem *p, uint32_t n);
