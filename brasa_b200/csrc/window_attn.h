// Windowed attention of a run of queries over the keys of a sequence (window_attn.cu). A key may come in two parts, one per key
// head and one shared by all heads; query heads may share key heads; the keys may lie one behind the other or in a ring.
#pragma once
#include "brasa_internal.h"

struct WindowAttn {
    const float *q;           // [tokens][ldq], head by head [dim own, rot shared part], not yet rotated
    const void *k, *v, *kr;   // rows of keys: [ldk] (kv_heads x kstep), [ldv] (kv_heads x vstep), [ldr], all rotated (kr unused with rot 0)
    const float *cos_t, *sin_t;  // [position][rot_dims / 2]
    const float *gate;        // [tokens][ldg], before the sigmoid; may be null
    void *out;                // [tokens][ldo] (heads x vdim)
    uint32_t ldq, ldk, ldv, ldr, ldg, ldo;
    uint32_t tokens, heads, dim, rot, rot_dims, vdim;  // the first rot_dims of the shared part are rotated; with rot 0, of the own part
    uint32_t pos0, key0, keys, window;  // a query sees its own position and the window - 1 before it
    float scale;
    uint32_t kv_heads, kstep, vstep;    // kstep, vstep: elements from one key head to the next (bf16: multiples of 8 reach the tensor cores)
    uint32_t ring;                      // 0: position p in row p - key0; otherwise in row p % ring (a multiple of 128; key0 then too)
    float softcap, out_scale;           // score <- softcap tanh(score / softcap) (0: as it is); the output is times out_scale
};
// f32: every buffer f32 and all arithmetic in f32; otherwise k, v, kr and out are bf16 (tcgen05 when the sizes allow). In a ring
// the rows of positions outside the range must hold finite values.
int32_t brasa_window_attention_launch(brasa_cmd *cmd, const WindowAttn &a, bool f32);
