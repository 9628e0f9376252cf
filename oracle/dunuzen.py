"""Plain float64 implementation of the Dunuzen design for tests: one function per mechanism, token by token where a
mechanism is a recurrence, whole score matrices where it is an attention. It shares no code with the product path.

A model is (config, weights): the parsed config.json and a dict name -> float array. `forward` takes the whole token
sequence of one request and returns logits for every position and the residual stream after every layer."""

from __future__ import annotations

import json
import pathlib
import struct

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, w, b, eps):
    c = x - np.mean(x, axis=-1, keepdims=True)
    return c / np.sqrt(np.mean(c * c, axis=-1, keepdims=True) + eps) * w + b


def unit(x, eps=1e-6):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + eps)


def rope_half(x, positions, dims, base):
    """Rotates the first `dims` entries of the last axis of x [tokens, ..., n]; entry i pairs with i + dims / 2."""
    half = dims // 2
    freq = float(base) ** (-2.0 * np.arange(half) / dims)
    a = np.asarray(positions, np.float64)[:, None] * freq
    a = a.reshape((a.shape[0],) + (1,) * (x.ndim - 2) + (half,))
    out = np.array(x, np.float64)
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * np.cos(a) - v * np.sin(a)
    out[..., half:dims] = v * np.cos(a) + u * np.sin(a)
    return out


def window_visible(n, size):
    """[n, n] mask: a query sees its own position and the size - 1 before it."""
    d = np.arange(n)[:, None] - np.arange(n)[None, :]
    return (d >= 0) & (d < size)


def softmax_rows(s, visible):
    s = np.where(visible, s, -np.inf)
    e = np.exp(s - np.max(s, axis=-1, keepdims=True))
    return e / np.sum(e, axis=-1, keepdims=True)


def latent_attention(h, W, m, eps):
    """h [tokens, width]; W(name) returns a tensor of this mixer; m the mixer's configuration."""
    n, H, d, r, dv, kr = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(n)
    q = (h @ W("q").T).reshape(n, H, d + r)
    down = h @ W("dkv").T
    c = rms(down[:, :kr], eps) * W("dkv.norm")
    k_rot = rope_half(down[:, kr:], pos, m["rot"]["dims"], m["rot"]["base"])
    q_rot = rope_half(q[..., d:], pos, m["rot"]["dims"], m["rot"]["base"])
    k = (c @ W("uk").T).reshape(n, H, d)
    v = (c @ W("uv").T).reshape(n, H, dv)
    gate = sigmoid(h @ W("g").T)
    seen = window_visible(n, m["mask"]["size"])
    out = np.zeros((n, H, dv))
    for head in range(H):
        s = (q[:, head, :d] @ k[:, head].T + q_rot[:, head] @ k_rot.T) * m["scale"]
        out[:, head] = softmax_rows(s, seen) @ v[:, head] * gate[:, head, None]
    return out.reshape(n, H * dv) @ W("o").T


def causal_conv(x, w):
    """Depthwise over time: x [tokens, channels], w [channels, taps], the last tap is the current token's."""
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    return sum(padded[i:i + x.shape[0]] * w[:, i] for i in range(taps))


def delta_decay(h, W, heads, dim):
    """The factor of every head and key channel, [tokens, heads, dim]."""
    z = softplus((h @ W("a1").T) @ W("a2").T + W("dt_bias")).reshape(h.shape[0], heads, dim)
    return np.exp(-np.exp(W("A_log"))[None, :, None] * z)


def delta_scan(q, k, v, g, beta, state):
    """One head: q, k, g [tokens, dim], v [tokens, vdim], beta [tokens]; returns outputs and the final state."""
    S, out = np.array(state, np.float64), []
    for t in range(q.shape[0]):
        S = g[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + np.outer(k[t], u)
        out.append(S.T @ q[t])
    return np.array(out).reshape(q.shape[0], v.shape[1]), S


def channel_delta(h, W, m, eps):
    n, H, KH, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(causal_conv(h @ W("q").T, W("q.conv"))).reshape(n, KH, d)
    k = silu(causal_conv(h @ W("k").T, W("k.conv"))).reshape(n, KH, d)
    v = silu(causal_conv(h @ W("v").T, W("v.conv"))).reshape(n, H, dv)
    q, k = unit(q) * d ** -0.5, unit(k)
    beta = sigmoid(h @ W("b").T)
    g = delta_decay(h, W, H, d)
    gate = sigmoid((h @ W("g1").T) @ W("g2").T).reshape(n, H, dv)
    o = np.zeros((n, H, dv))
    for head in range(H):
        kh = head // (H // KH)
        o[:, head], _ = delta_scan(q[:, kh], k[:, kh], v[:, head], g[:, head], beta[:, head], np.zeros((d, dv)))
    o = rms(o, eps) * W("norm") * gate
    return o.reshape(n, H * dv) @ W("o").T


def feed_forward(h, W):
    return np.maximum(h @ W("up").T + W("up.b"), 0.0) ** 2 @ W("down").T + W("down.b")


MIXERS = {"latent_attention": latent_attention, "channel_delta": channel_delta}


def forward(config, weights, tokens):
    """Returns (logits [tokens, vocab], residual stream after every layer [layers, tokens, width])."""
    eps = config["norm"]["eps"]
    T = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    x = T["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    after = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](layer_norm(x, T[p + "norm1"], T[p + "norm1.b"], eps), lambda s: T[p + "mix." + s], layer["mixer"], eps)
        if layer["mlp"] is not None:
            y = y + feed_forward(layer_norm(x, T[p + "norm2"], T[p + "norm2.b"], eps), lambda s: T[p + "mlp." + s])
        x = x + y
        after.append(x)
    x = layer_norm(x, T["final.norm"], T["final.norm.b"], eps)
    return x @ T["head"].T * config["logit_scale"], np.array(after)


# ---- files ------------------------------------------------------------------------------------------


def bf16_bits(x):
    """float array -> bfloat16 bit patterns, round to nearest even."""
    b = np.ascontiguousarray(x, np.float32).view(np.uint32)
    return ((b + 0x7FFF + ((b >> 16) & 1)) >> 16).astype(np.uint16)


def bf16_round(x):
    return (bf16_bits(x).astype(np.uint32) << 16).view(np.float32)


def read_safetensors(path):
    raw = pathlib.Path(path).read_bytes()
    n = struct.unpack("<Q", raw[:8])[0]
    out = {}
    for name, t in json.loads(raw[8:8 + n]).items():
        if name == "__metadata__":
            continue
        b, e = t["data_offsets"]
        data = raw[8 + n + b:8 + n + e]
        if t["dtype"] == "BF16":
            out[name] = (np.frombuffer(data, "<u2").astype(np.uint32) << 16).view(np.float32).reshape(t["shape"])
        else:
            out[name] = np.frombuffer(data, {"F32": "<f4", "I32": "<i4"}[t["dtype"]]).reshape(t["shape"])
    return out


def write_model(folder, config, weights):
    """config.json and a bfloat16 model.safetensors."""
    folder = pathlib.Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config))
    header, blobs, at = {}, [], 0
    for name, w in weights.items():
        data = bf16_bits(w).tobytes()
        header[name] = {"dtype": "BF16", "shape": list(np.shape(w)), "data_offsets": [at, at + len(data)]}
        at += len(data)
        blobs.append(data)
    h = json.dumps(header).encode()
    h += b" " * (-len(h) % 8)
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(h)) + h + b"".join(blobs))


def tensor_shapes(config, ranks=None):
    """name -> shape of every tensor. ranks[layer] = (inner size of the decay projection, of the gate projection)."""
    w = config["width"]
    out = {"embed": (config["vocab"], w)}
    for i, layer in enumerate(config["layers"]):
        m, p = layer["mixer"], f"l{i}."
        for nm in ("norm1", "norm2") if layer["mlp"] is not None else ("norm1",):
            out[p + nm] = out[p + nm + ".b"] = (w,)
        x = p + "mix."
        if layer["type"] == "latent_attention":
            H, r, kr = m["heads"], m["rot_dim"], m["kv_rank"]
            out |= {x + "q": (H * (m["dim"] + r), w), x + "dkv": (kr + r, w), x + "dkv.norm": (kr,), x + "uk": (H * m["dim"], kr),
                    x + "uv": (H * m["vdim"], kr), x + "g": (H, w), x + "o": (w, H * m["vdim"])}
        else:
            H, qk, vd = m["heads"], m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            ra, rg = (ranks or {}).get(i, (20, 12))
            out |= {x + "q": (qk, w), x + "q.conv": (qk, m["conv"]), x + "k": (qk, w), x + "k.conv": (qk, m["conv"]), x + "v": (vd, w),
                    x + "v.conv": (vd, m["conv"]), x + "b": (H, w), x + "A_log": (H,), x + "norm": (m["vdim"],), x + "a1": (ra, w),
                    x + "a2": (H * m["dim"], ra), x + "dt_bias": (H * m["dim"],), x + "g1": (rg, w), x + "g2": (vd, rg), x + "o": (w, vd)}
        if layer["mlp"] is not None:
            f = layer["mlp"]["ff"]
            y = p + "mlp."
            out |= {y + "up": (f, w), y + "up.b": (f,), y + "down": (w, f), y + "down.b": (w,)}
    out |= {"final.norm": (w,), "final.norm.b": (w,), "head": (config["vocab"], w)}
    return out


def random_weights(config, seed, ranks=None):
    """Random bfloat16-representable weights whose norms, biases, decays and convolutions are all away from 0 and 1."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config, ranks).items():
        z = rng.standard_normal(shape)
        leaf = name.split(".")[-1]
        if name == "embed":
            w = z / config["embedding"]["scale"]
        elif leaf.startswith("norm"):
            w = 1.0 + 0.3 * z
        elif name.endswith(("norm1.b", "norm2.b", "final.norm.b", "up.b", "down.b")):
            w = 0.3 * z
        elif leaf == "conv":
            w = 0.6 * z
        elif leaf == "A_log":
            w = -1.0 + z
        elif leaf == "dt_bias":
            w = -2.0 + z
        elif leaf in ("a1", "a2"):
            w = 1.5 * z / np.sqrt(shape[1])
        else:
            w = z / np.sqrt(shape[1])
        out[name] = bf16_round(w)
    return out
