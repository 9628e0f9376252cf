"""Small Dunuzen configurations for the tests: sizes that divide nothing, sizes the tensor-core kernels take, and sizes of one."""

import numpy as np

from oracle import dunuzen as D


def latent(heads, dim, rot, vdim, kv_rank, window, base=1000.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window}, "rot": {"base": base, "dims": rot},
            "scale": scale or (dim + rot) ** -0.5}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def config(width, vocab, layers, eps=1e-5, embed=1.0, logit=1.0):
    """layers: (type, mixer, ff or None)"""
    return {"architecture": "Dunuzen", "vocab": vocab, "width": width, "embedding": {"scale": embed}, "norm": {"eps": eps}, "logit_scale": logit,
            "layers": [{"type": t, "mixer": m, "mlp": {"kind": "dense", "ff": f} if f else None} for t, m, f in layers]}


LA, CD = "latent_attention", "channel_delta"
CASES = {
    # no size is a multiple of eight: padded weights, the fallback attention; two windows, two rotations, a layer without feed-forward
    "ragged": (config(100, 93, [(CD, delta(6, 3, 20, 36, 3), 70), (LA, latent(3, 20, 12, 28, 44, 19, 500.0), 121), (LA, latent(5, 12, 6, 12, 30, 50, 20000.0), None),
                                (CD, delta(2, 1, 70, 18, 5), 33)], eps=3e-4, embed=2.5, logit=0.5), {0: (10, 7), 3: (3, 13)}),
    # tensor-core attention with one and two 64-wide blocks of key and value dimensions
    "tiles": (config(128, 200, [(LA, latent(4, 32, 8, 48, 64, 130), 96), (CD, delta(4, 4, 64, 64, 4), 256), (LA, latent(2, 96, 32, 96, 136, 64), 64),
                                (LA, latent(3, 136, 16, 64, 96, 300), 40)], embed=3.0), {1: (16, 24)}),
    # the smallest of everything: one head, a window of one token, a convolution of one tap
    "ones": (config(24, 40, [(LA, latent(1, 8, 2, 8, 8, 1), 8), (CD, delta(1, 1, 4, 4, 1), 16), (CD, delta(3, 1, 8, 16, 2), None)]), {1: (1, 1), 2: (2, 2)}),
    # a state wider than the decode kernel keeps in registers
    "wide": (config(64, 50, [(CD, delta(2, 1, 136, 144, 4), 32), (LA, latent(2, 16, 8, 16, 16, 7), 32)]), {0: (9, 20)}),
}


def build(name, seed=0, peak=4.0):
    """(config, weights): `peak` scales the attention queries, so that single keys dominate and a wrong one shows."""
    cfg, ranks = CASES[name]
    w = D.random_weights(cfg, seed, ranks)
    for i, layer in enumerate(cfg["layers"]):
        if layer["type"] == LA:
            w[f"l{i}.mix.q"] = D.bf16_round(w[f"l{i}.mix.q"] * peak)
    return cfg, w


def tokens(cfg, n, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], size=n).astype(np.uint32)


def off(got, want):
    """Worst row: root mean square of the difference over that of the wanted row's deviations."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    return float(np.max(np.sqrt((d ** 2).mean(-1)) / np.std(want, axis=-1)))
