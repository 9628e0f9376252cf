"""Small Gugedra configurations for the tests: sizes that divide nothing, sizes the tensor-core kernels take, sizes of one, and
sizes beyond the fast kernels."""

from oracle import dunuzen as D
from oracle import gugedra as G


def attn(heads, kv_heads, dim, vdim, window, rot, base=1000.0, scale=None, softcap=20.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "rot": {"base": base, "dims": rot},
            "scale": scale or dim ** -0.5, "softcap": softcap}


def ssm(heads, vdim, state, groups, norm_groups, conv):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}


def parallel(left, right, left_scale=0.8, right_scale=1.3):
    return {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def config(width, vocab, layers, eps=1e-5, side=8, cap=25.0):
    """layers: (mixer, ff or None); a mixer with a left side is a parallel one"""
    return {"architecture": "Gugedra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "token_side": {"dim": side}, "logit_softcap": cap,
            "layers": [{"type": "parallel" if "left" in m else "delta", "mixer": m, "mlp": {"kind": "dense", "ff": f} if f else None} for m, f in layers]}


CASES = {
    # no size is a multiple of eight: padded weights and heads; two windows, two rotations, with and without feed-forward, three taps and five
    "ragged": config(100, 93, [(delta(6, 3, 20, 36, 3), 70), (parallel(attn(6, 2, 20, 12, 19, 10, 500.0), ssm(6, 20, 13, 3, 2, 4)), 121),
                               (parallel(attn(5, 5, 13, 30, 50, 12, 20000.0, 0.4, 7.0), ssm(4, 33, 70, 2, 12, 5), 1.7, 0.3), None),
                               (delta(2, 1, 70, 18, 5), None)], eps=3e-4, side=5, cap=9.0),
    # every width of the tensor-core attention's key and value blocks, state products with one and more blocks of value columns
    "tiles": config(128, 200, [(parallel(attn(8, 2, 64, 128, 130, 64), ssm(8, 64, 128, 1, 1, 4)), 96), (delta(4, 4, 64, 64, 4), 256),
                               (parallel(attn(4, 1, 128, 64, 64, 32), ssm(2, 128, 64, 2, 4, 2), 1.0, 1.0), 64),
                               (parallel(attn(2, 2, 192, 72, 300, 16, softcap=40.0), ssm(6, 16, 200, 3, 3, 4)), 40), (delta(2, 2, 128, 96, 4), None)]),
    # the smallest of everything: one head, a window of one token, one state, convolutions of one tap (a large eps: norms of single
    # values are signs otherwise)
    "ones": config(24, 40, [(parallel(attn(1, 1, 2, 1, 1, 2), ssm(1, 1, 1, 1, 1, 1)), 1), (delta(1, 1, 4, 4, 1), 3), (delta(3, 1, 8, 16, 2), None),
                            (parallel(attn(3, 1, 8, 8, 2, 8), ssm(2, 8, 16, 2, 2, 2)), None)], eps=0.1, side=1),
    # beyond the fast kernels: wide heads, a softcap whose exponentials need a moving reference, states wider than the products take
    "wide": config(64, 50, [(parallel(attn(10, 1, 200, 136, 33, 100, softcap=90.0), ssm(2, 20, 300, 1, 1, 4)), 32), (delta(2, 1, 136, 144, 4), 32),
                            (parallel(attn(2, 2, 16, 200, 7, 4), ssm(1, 150, 24, 1, 5, 3)), 32)]),
}


def build(name, seed=0, peak=5.0):
    """(config, weights): `peak` scales the attention queries, so that single keys dominate and a wrong one shows."""
    cfg = CASES[name]
    w = G.random_weights(cfg, seed)
    for i, layer in enumerate(cfg["layers"]):
        if layer["type"] == "parallel":
            w[f"l{i}.mix.left.q"] = D.bf16_round(w[f"l{i}.mix.left.q"] * peak)
    return cfg, w
