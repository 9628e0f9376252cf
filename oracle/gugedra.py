"""Plain float64 implementation of the Gugedra design for tests: one function per mechanism, token by token where a mechanism is
a recurrence, whole score matrices where it is an attention. It shares no code with the product path.

A model is (config, weights): the parsed config.json and a dict name -> float array. `forward` takes the whole token
sequence of one request and returns logits for every position and the residual stream after every layer. `r` rounds what a
16-bit implementation may keep in 16 bits (the products' inputs, keys, values, convolved values); with bf16_round it tells how far
rounding alone carries a model."""

from __future__ import annotations

import numpy as np

from .dunuzen import bf16_round, causal_conv, delta_scan, rms, rope_half, sigmoid, silu, softmax_rows, softplus, unit, window_visible


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def softcap(z, cap):
    return cap * np.tanh(z / cap)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def grouped_rms(x, groups, eps):
    """Equal parts of the last axis, each over its own root mean square."""
    return rms(x.reshape(x.shape[:-1] + (groups, -1)), eps).reshape(x.shape)


def attention_scores(q, k, scale, cap):
    """q [n, dim], k [n, dim] of one head, both rotated."""
    return softcap(q @ k.T * scale, cap)


def exact(x):
    return x


def window_attention(h, W, m, r=exact):
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos, dims, base = np.arange(n), m["rot"]["dims"], m["rot"]["base"]
    q = r(rope_half((h @ W("q").T).reshape(n, H, d), pos, dims, base))
    k = r(rope_half((h @ W("k").T).reshape(n, G, d), pos, dims, base))
    v = r((h @ W("v").T).reshape(n, G, dv))
    seen = window_visible(n, m["mask"]["size"])
    out = np.zeros((n, H, dv))
    for head in range(H):
        g = head // (H // G)
        out[:, head] = softmax_rows(attention_scores(q[:, head], k[:, g], m["scale"], m["softcap"]), seen) @ v[:, g]
    return r(out.reshape(n, H * dv)) @ W("o").T


def state_space_scan(x, B, C, dt, a_log, D, state):
    """One head: x [tokens, vdim], B and C [tokens, state], dt [tokens]; returns outputs and the final state [state, vdim]."""
    S, out = np.array(state, np.float64), []
    for t in range(x.shape[0]):
        S = np.exp(-np.exp(a_log) * dt[t]) * S + dt[t] * np.outer(B[t], x[t])
        out.append(S.T @ C[t] + D * x[t])
    return np.array(out).reshape(x.shape), S


def state_space(h, W, m, eps, r=exact):
    n, H, dv, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    p = h @ W("in").T
    z, conv_in, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    c = r(silu(causal_conv(conv_in, W("conv")) + W("conv.b")))
    x, B, C = c[:, :inner].reshape(n, H, dv), c[:, inner:inner + G * N].reshape(n, G, N), c[:, inner + G * N:].reshape(n, G, N)
    dt = softplus(dt + W("dt_bias"))
    y = np.zeros((n, H, dv))
    for head in range(H):
        g = head // (H // G)
        y[:, head], _ = state_space_scan(x[:, head], B[:, g], C[:, g], dt[:, head], W("A_log")[head], W("D")[head], np.zeros((N, dv)))
    y = y.reshape(n, inner) * silu(z)
    return r(grouped_rms(y, m["norm_groups"], eps) * W("norm")) @ W("o").T


def parallel(h, W, m, eps, r=exact):
    return (m["left_scale"] * window_attention(h, lambda s: W("left." + s), m["left"], r)
            + m["right_scale"] * state_space(h, lambda s: W("right." + s), m["right"], eps, r))


def delta(h, W, m, eps, r=exact):
    n, H, KH, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(causal_conv(h @ W("q").T, W("q.conv"))).reshape(n, KH, d)
    k = silu(causal_conv(h @ W("k").T, W("k.conv"))).reshape(n, KH, d)
    v = silu(causal_conv(h @ W("v").T, W("v.conv"))).reshape(n, H, dv)
    q, k = unit(q) * d ** -0.5, unit(k)
    beta = sigmoid(h @ W("b").T)
    g = np.exp(-np.exp(W("A_log")) * softplus(h @ W("a").T + W("dt_bias")))
    o = np.zeros((n, H, dv))
    for head in range(H):
        kh = head // (H // KH)
        decay = np.repeat(g[:, head, None], d, axis=1)
        o[:, head], _ = delta_scan(q[:, kh], k[:, kh], v[:, head], decay, beta[:, head], np.zeros((d, dv)))
    o = rms(o, eps) * W("norm") * silu((h @ W("g").T).reshape(n, H, dv))
    return r(o.reshape(n, H * dv)) @ W("o").T


def feed_forward(h, W, r=exact):
    return r(silu(h @ W("gate").T) * (h @ W("up").T)) @ W("down").T


def token_side(x, e, W, eps, r=exact):
    """x [tokens, width], e [tokens, dim]: this layer's part of the tokens' second embedding."""
    y = r(gelu_tanh(r(x) @ W("gate").T) * e) @ W("proj").T
    return rms_norm(y, W("norm"), eps)


MIXERS = {"parallel": parallel, "delta": delta}


def layer(x, e, cfg, entry, W, r=exact):
    """One layer on the residual stream x; W(name) returns a tensor of this layer."""
    eps = cfg["norm"]["eps"]
    y = MIXERS[entry["type"]](r(rms_norm(x, W("norm1"), eps)), lambda s: W("mix." + s), entry["mixer"], eps, r)
    x = x + rms_norm(y, W("norm1b"), eps)
    if entry["mlp"] is not None:
        x = x + rms_norm(feed_forward(r(rms_norm(x, W("norm2"), eps)), lambda s: W("mlp." + s), r), W("norm2b"), eps)
    return x + token_side(x, e, lambda s: W("side." + s), eps, r)


def forward(config, weights, tokens, r=exact):
    """Returns (logits [tokens, vocab], residual stream after every layer [layers, tokens, width])."""
    T = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    ids, dim, after = np.asarray(tokens), config["token_side"]["dim"], []
    x = T["embed"][ids]
    for i, entry in enumerate(config["layers"]):
        x = layer(x, T["side.embed"][ids][:, i * dim:(i + 1) * dim], config, entry, lambda s: T[f"l{i}." + s], r)
        after.append(x)
    x = rms_norm(x, T["final.norm"], config["norm"]["eps"])
    return softcap(r(x) @ T["head"].T, config["logit_softcap"]), np.array(after)


def tensor_shapes(config):
    """name -> shape of every tensor."""
    w, L, sd = config["width"], len(config["layers"]), config["token_side"]["dim"]
    out = {"embed": (config["vocab"], w), "side.embed": (config["vocab"], L * sd)}
    for i, entry in enumerate(config["layers"]):
        m, p = entry["mixer"], f"l{i}."
        for nm in ("norm1", "norm1b") + (("norm2", "norm2b") if entry["mlp"] is not None else ()):
            out[p + nm] = (w,)
        x = p + "mix."
        if entry["type"] == "parallel":
            a, r = m["left"], m["right"]
            inner, gn = r["heads"] * r["vdim"], r["groups"] * r["state"]
            out |= {x + "left.q": (a["heads"] * a["dim"], w), x + "left.k": (a["kv_heads"] * a["dim"], w), x + "left.v": (a["kv_heads"] * a["vdim"], w),
                    x + "left.o": (w, a["heads"] * a["vdim"]), x + "right.in": (2 * inner + 2 * gn + r["heads"], w),
                    x + "right.conv": (inner + 2 * gn, r["conv"]), x + "right.conv.b": (inner + 2 * gn,), x + "right.dt_bias": (r["heads"],),
                    x + "right.A_log": (r["heads"],), x + "right.D": (r["heads"],), x + "right.norm": (inner,), x + "right.o": (w, inner)}
        else:
            H, qk, vd = m["heads"], m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            out |= {x + "q": (qk, w), x + "q.conv": (qk, m["conv"]), x + "k": (qk, w), x + "k.conv": (qk, m["conv"]), x + "v": (vd, w),
                    x + "v.conv": (vd, m["conv"]), x + "b": (H, w), x + "A_log": (H,), x + "norm": (m["vdim"],), x + "a": (H, w),
                    x + "dt_bias": (H,), x + "g": (vd, w), x + "o": (w, vd)}
        if entry["mlp"] is not None:
            f = entry["mlp"]["ff"]
            out |= {p + "mlp.gate": (f, w), p + "mlp.up": (f, w), p + "mlp.down": (w, f)}
        out |= {p + "side.gate": (sd, w), p + "side.proj": (w, sd), p + "side.norm": (w,)}
    return out | {"final.norm": (w,), "head": (config["vocab"], w)}


def random_weights(config, seed):
    """Random bfloat16-representable weights whose norms, biases, decays and convolutions are all away from 0 and 1."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        z = rng.standard_normal(shape)
        leaf = name.split(".")[-1]
        if name in ("embed", "side.embed"):
            w = z
        elif leaf.startswith("norm"):
            w = 1.0 + 0.3 * z
        elif leaf == "conv":
            w = 0.6 * z
        elif name.endswith("conv.b"):
            w = 0.3 * z
        elif leaf == "A_log":
            w = -1.0 + z
        elif leaf == "dt_bias":
            w = -1.5 + z
        elif leaf == "D":
            w = 1.0 + 0.5 * z
        else:
            w = z / np.sqrt(shape[1])
        out[name] = bf16_round(w)
    return out
