// Windowed attention of a run of queries over a contiguous range of keys, for keys that come in two parts: one per head and
// one shared by all heads (window_attn.cu).
#pragma once
#include "brasa_internal.h"

struct WindowAttn {
    const float *q;           // [tokens][ldq], head by head [dim unrotated, rot rotated], not yet rotated
    const void *k, *v, *kr;   // rows of positions key0 ..: [keys][ldk] (heads x dim), [keys][ldv] (heads x vdim), [keys][ldr] (rotated)
    const float *cos_t, *sin_t;  // [position][rot_dims / 2]
    const float *gate;        // [tokens][ldg], before the sigmoid
    void *out;                // [tokens][ldo] (heads x vdim)
    uint32_t ldq, ldk, ldv, ldr, ldg, ldo;
    uint32_t tokens, heads, dim, rot, rot_dims, vdim;
    uint32_t pos0, key0, keys, window;  // a query sees its own position and the window - 1 before it
    float scale;
};
// f32: every buffer f32 and all arithmetic in f32; otherwise k, v, kr and out are bf16 (tcgen05 when the sizes allow).
int32_t brasa_window_attention_launch(brasa_cmd *cmd, const WindowAttn &a, bool f32);
