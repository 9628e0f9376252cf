"""Synthetic random-init Qwen3 models in the `.brasa` container, generated and quantised on the GPU.

The benchmark configurations call for weights drawn N(0, 0.02) from a seed with norm vectors at 1 and
the `.brasa` quantisation (linear layers q4_0, embedding table q6_0, norms f32). This module is the
device-side converter for that case: values come from brasa_k_randn, blocks from brasa_k_quantize
(bit-identical to crates/quant/src/convert.rs:70-151), and the container is laid out exactly like
tools/convert_brasa.py:92-170 writes it (sorted names, 16 KiB pages, per-tensor sha256).
"""

from __future__ import annotations

import hashlib
import json
import pathlib
import struct

import numpy as np

from . import Context, Kernels, WeightType

PAGE = 16384
QWEN3_4B = {"model_type": "qwen3", "tie_word_embeddings": True, "num_hidden_layers": 36, "hidden_size": 2560,
            "intermediate_size": 9728, "num_attention_heads": 32, "num_key_value_heads": 8, "head_dim": 128,
            "rms_norm_eps": 1e-6, "rope_theta": 1e6, "vocab_size": 151936, "max_position_embeddings": 40960}
QWEN3_32B = {"model_type": "qwen3", "tie_word_embeddings": False, "num_hidden_layers": 64, "hidden_size": 5120,
             "intermediate_size": 25600, "num_attention_heads": 64, "num_key_value_heads": 8, "head_dim": 128,
             "rms_norm_eps": 1e-6, "rope_theta": 1e6, "vocab_size": 151936, "max_position_embeddings": 40960}
_BLOCK_BYTES = {"q4_0": 18, "q6_0": 26, "q8_0": 34}
_QT = {"q4_0": WeightType.Q4_0, "q6_0": WeightType.Q6_0, "q8_0": WeightType.Q8_0}


def tensor_shapes(cfg: dict) -> dict[str, list[int]]:
    H, F, V, D = cfg["hidden_size"], cfg["intermediate_size"], cfg["vocab_size"], cfg["head_dim"]
    qd, kvd = cfg["num_attention_heads"] * D, cfg["num_key_value_heads"] * D
    t = {"model.embed_tokens.weight": [V, H], "model.norm.weight": [H]}
    for i in range(cfg["num_hidden_layers"]):
        p = f"model.layers.{i}."
        t.update({p + "input_layernorm.weight": [H], p + "post_attention_layernorm.weight": [H],
                  p + "self_attn.q_norm.weight": [D], p + "self_attn.k_norm.weight": [D],
                  p + "self_attn.q_proj.weight": [qd, H], p + "self_attn.k_proj.weight": [kvd, H],
                  p + "self_attn.v_proj.weight": [kvd, H], p + "self_attn.o_proj.weight": [H, qd],
                  p + "mlp.gate_proj.weight": [F, H], p + "mlp.up_proj.weight": [F, H], p + "mlp.down_proj.weight": [H, F]})
    if not cfg.get("tie_word_embeddings", True):
        t["lm_head.weight"] = [cfg.get("tp_head_rows", V), H]  # a tensor-parallel shard holds its rows of the vocabulary
    return t


def dtype_for(name: str, ndim: int) -> str:
    if ndim == 1:
        return "f32"
    return "q6_0" if name == "model.embed_tokens.weight" else "q4_0"


def _nbytes(dtype: str, shape) -> int:
    n = int(np.prod(shape))
    return 4 * n if dtype == "f32" else n // 32 * _BLOCK_BYTES[dtype]


def _header(meta: dict) -> bytes:
    js = json.dumps(meta, ensure_ascii=False, separators=(",", ":")).encode()
    return b"BRSA" + struct.pack("<IQ", 1, len(js)) + js


def write_synthetic_model(ctx: Context, path, cfg: dict, seed: int = 0, std: float = 0.02) -> dict:
    """Writes `path` (model.brasa) with seeded N(0, std) matrices and norm vectors of ones."""
    path = pathlib.Path(path)
    K = Kernels(ctx)
    shapes = tensor_shapes(cfg)
    tensors = []
    for name in sorted(shapes):
        dt = dtype_for(name, len(shapes[name]))
        tensors.append({"name": name, "dtype": dt, "shape": shapes[name], "nbytes": _nbytes(dt, shapes[name]), "offset": 0,
                        "sha256": "0" * 64})
    meta = {"format": "brasa", "version": 1, "converter": "brasa_b200.synth",
            "model": {"family": "qwen3", "source_repo": "synthetic", "source_commit": f"seed-{seed}", "config": cfg},
            "quant": {"block": 32, "scheme": "q4_0 linears, q6_0 embeddings/lm_head, f32 norms"},
            "page": PAGE, "tensors": tensors, "data_sha256": "0" * 64}
    data_start = PAGE
    while True:
        off = data_start
        for t in tensors:
            t["offset"] = off
            off = (off + t["nbytes"] + PAGE - 1) // PAGE * PAGE
        if len(_header(meta)) <= data_start:
            break
        data_start += PAGE
    total, provisional = off, len(_header(meta))
    biggest = max(int(np.prod(t["shape"])) for t in tensors if t["dtype"] != "f32")
    f32buf = ctx.buffer(biggest * 4)
    qbuf = ctx.buffer(max(t["nbytes"] for t in tensors))
    stream_off = 0
    # a tensor-parallel shard (brasa_b200.tp.shard_config): the replicated embedding table comes from the shared seed,
    # everything else from a seed of the rank's own
    own_seed = seed + 1000003 * (cfg["tp_rank"] + 1) if "tp_rank" in cfg else seed
    with open(path, "wb") as f:
        f.truncate(total)
        for t in tensors:
            n = int(np.prod(t["shape"]))
            if t["dtype"] == "f32":
                data = np.ones(n, dtype="<f4").tobytes()
            else:
                cmd = ctx.command()
                shared = "tp_rank" in cfg and t["name"] == "model.embed_tokens.weight"
                K.randn(cmd, f32buf, n, seed if shared else own_seed, 0 if shared else stream_off, std)
                K.quantize(cmd, _QT[t["dtype"]], f32buf, qbuf, n)
                cmd.wait()
                data = qbuf.download(np.uint8, t["nbytes"]).tobytes()
                stream_off += 0 if shared else (n + 1) // 2
            t["sha256"] = hashlib.sha256(data).hexdigest()
            f.seek(t["offset"])
            f.write(data)
        meta["data_sha256"] = hashlib.sha256("".join(t["sha256"] for t in tensors).encode()).hexdigest()
        header = _header(meta)
        assert len(header) == provisional
        f.seek(0)
        f.write(header)
    f32buf.free()
    qbuf.free()
    return meta


def weight_bytes_per_token(cfg: dict) -> int:
    """Bytes of weights one decode token reads: every quantised matrix once, norm vectors, one embedding row."""
    total = 0
    for name, shape in tensor_shapes(cfg).items():
        dt = dtype_for(name, len(shape))
        if name == "model.embed_tokens.weight" and not cfg.get("tie_word_embeddings", True):
            continue
        total += _nbytes(dt, shape)
    total += cfg["hidden_size"] // 32 * 26  # the embedding row of the input token
    return total


def kv_bytes_per_position(cfg: dict, kv: str = "f16") -> int:
    rows = 2 * cfg["num_hidden_layers"] * cfg["num_key_value_heads"]
    return rows * {"f32": 512, "f16": 256, "q8_0": 136}[kv]


# ---- layer-stack models: config.json + model.safetensors with seeded bf16 weights, drawn on the host ---------------------


def dunuzen_config(width: int, ff: int, heads: int, kv_heads: int, layers: list[str], vocab: int, window: int, dim: int = 128, rot_dim: int = 64,
                   vdim: int = 128, kv_rank: int = 512, conv: int = 4) -> dict:
    """A configuration of uniform layers; `layers` names the mixer of each."""
    mixers = {"latent_attention": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window},
                                   "rot": {"base": 10000.0, "dims": rot_dim}, "scale": (dim + rot_dim) ** -0.5},
              "channel_delta": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}
    return {"architecture": "Dunuzen", "vocab": vocab, "width": width, "embedding": {"scale": 1.0}, "norm": {"eps": 1e-5}, "logit_scale": 1.0,
            "layers": [{"type": t, "mixer": mixers[t], "mlp": {"kind": "dense", "ff": ff}} for t in layers]}


def dunuzen_shapes(cfg: dict, rank: int = 128) -> dict[str, list[int]]:
    """name -> shape; rank: inner size of the decay's and the output gate's projections."""
    w, t = cfg["width"], {"embed": [cfg["vocab"], cfg["width"]]}
    for i, layer in enumerate(cfg["layers"]):
        m, p, x = layer["mixer"], f"l{i}.", f"l{i}.mix."
        for n in ("norm1", "norm2"):
            t.update({p + n: [w], p + n + ".b": [w]})
        if layer["type"] == "latent_attention":
            h, kr = m["heads"], m["kv_rank"]
            t.update({x + "q": [h * (m["dim"] + m["rot_dim"]), w], x + "dkv": [kr + m["rot_dim"], w], x + "dkv.norm": [kr], x + "uk": [h * m["dim"], kr],
                      x + "uv": [h * m["vdim"], kr], x + "g": [h, w], x + "o": [w, h * m["vdim"]]})
        else:
            h, qk, vd = m["heads"], m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            t.update({x + "q": [qk, w], x + "q.conv": [qk, m["conv"]], x + "k": [qk, w], x + "k.conv": [qk, m["conv"]], x + "v": [vd, w],
                      x + "v.conv": [vd, m["conv"]], x + "b": [h, w], x + "A_log": [h], x + "norm": [m["vdim"]], x + "a1": [rank, w],
                      x + "a2": [h * m["dim"], rank], x + "dt_bias": [h * m["dim"]], x + "g1": [rank, w], x + "g2": [vd, rank], x + "o": [w, vd]})
        f = layer["mlp"]["ff"]
        t.update({p + "mlp.up": [f, w], p + "mlp.up.b": [f], p + "mlp.down": [w, f], p + "mlp.down.b": [w]})
    t.update({"final.norm": [w], "final.norm.b": [w], "head": [cfg["vocab"], w]})
    return t


def write_synthetic_stack(folder, cfg: dict, shapes: dict[str, list[int]], seed: int = 0, std: float = 0.02) -> None:
    """Seeded N(0, std) matrices, norm weights of ones, biases of zeros; drawn and rounded tensor by tensor in parallel."""
    import concurrent.futures
    import os
    folder = pathlib.Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    header, at = {}, 0
    for name, shape in shapes.items():
        n = 2 * int(np.prod(shape))
        header[name] = {"dtype": "BF16", "shape": shape, "data_offsets": [at, at + n]}
        at += n
    js = json.dumps(header).encode()
    js += b" " * (-len(js) % 8)

    def draw(item):
        i, (name, shape) = item
        if len(shape) == 1:
            w = np.full(shape, 1.0 if "norm" in name and not name.endswith(".b") else (-1.0 if name.endswith("dt_bias") else 0.0), np.float32)
        else:
            w = np.random.Generator(np.random.SFC64([seed, i])).standard_normal(shape, dtype=np.float32)
            w *= np.float32(0.5 if name.endswith(".conv") else std)
        b = w.view(np.uint32)
        return name, ((b + np.uint32(0x8000)) >> np.uint32(16)).astype("<u2")

    tmp = folder / f"model.safetensors.{os.getpid()}.tmp"
    with open(tmp, "wb") as f, concurrent.futures.ThreadPoolExecutor(max_workers=min(16, os.cpu_count() or 1)) as ex:
        f.write(struct.pack("<Q", len(js)) + js)
        for name, data in ex.map(draw, enumerate(shapes.items())):
            f.seek(8 + len(js) + header[name]["data_offsets"][0])
            f.write(data.tobytes())
    os.replace(tmp, folder / "model.safetensors")
    (folder / "config.json").write_text(json.dumps(cfg))


def dunuzen_decode_bytes(cfg: dict, pos: int, rank: int = 128) -> int:
    """Bytes one bf16 decode step at position pos has to move: every matrix once, the states read and written, the visible rows."""
    total = 2 * sum(int(np.prod(s)) for n, s in dunuzen_shapes(cfg, rank).items() if n != "embed") + 2 * cfg["width"]
    for layer in cfg["layers"]:
        m = layer["mixer"]
        if layer["type"] == "latent_attention":
            total += 2 * min(pos + 1, m["mask"]["size"]) * (m["kv_rank"] + m["rot_dim"])
        else:
            total += 8 * m["heads"] * m["dim"] * m["vdim"]
    return total


def dunuzen_prefill_flops(cfg: dict, tokens: int, rank: int = 128) -> dict:
    """Operations of a prompt of `tokens` tokens: products with weights, attention inside the window, delta rule."""
    mm = sum(2 * tokens * int(np.prod(s)) for n, s in dunuzen_shapes(cfg, rank).items() if len(s) == 2 and n not in ("embed", "head") and not n.endswith(".conv"))
    attn = delta = 0
    for layer in cfg["layers"]:
        m = layer["mixer"]
        if layer["type"] == "latent_attention":
            w = min(m["mask"]["size"], tokens)
            pairs = w * (w + 1) // 2 + (tokens - w) * w
            attn += 2 * pairs * m["heads"] * (m["dim"] + m["rot_dim"] + m["vdim"])
        else:
            delta += 7 * tokens * m["heads"] * m["dim"] * m["vdim"]
    return {"matmul": mm, "attention": attn, "delta": delta}


def gugedra_config(width: int, ff: int, heads: int, kv_heads: int, layers: list[str], vocab: int, window: int, dim: int = 128, rot_dims: int = 64, vdim: int = 128,
                   state: int = 128, ssm_vdim: int = 64, conv: int = 4, side: int = 256) -> dict:
    """A configuration of uniform layers; `layers` names the mixer of each. The state-space side is twice as wide as the model."""
    ssm_heads = 2 * width // ssm_vdim
    mixers = {"parallel": {"left": {"heads": heads, "kv_heads": max(1, heads // 4), "dim": dim, "vdim": vdim, "mask": {"size": window},
                                    "rot": {"base": 10000.0, "dims": rot_dims}, "scale": dim ** -0.5, "softcap": 50.0},
                           "right": {"heads": ssm_heads, "vdim": ssm_vdim, "state": state, "groups": 1, "norm_groups": 1, "conv": conv},
                           "left_scale": 1.0, "right_scale": 1.0},
              "delta": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}
    return {"architecture": "Gugedra", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "token_side": {"dim": side}, "logit_softcap": 30.0,
            "layers": [{"type": t, "mixer": mixers[t], "mlp": {"kind": "dense", "ff": ff}} for t in layers]}


def gugedra_shapes(cfg: dict) -> dict[str, list[int]]:
    w, side = cfg["width"], cfg["token_side"]["dim"]
    t = {"embed": [cfg["vocab"], w], "side.embed": [cfg["vocab"], side * len(cfg["layers"])]}
    for i, layer in enumerate(cfg["layers"]):
        m, p, x = layer["mixer"], f"l{i}.", f"l{i}.mix."
        t.update({p + n: [w] for n in ("norm1", "norm1b", "norm2", "norm2b")})
        if layer["type"] == "parallel":
            a, r = m["left"], m["right"]
            inner, gn = r["heads"] * r["vdim"], r["groups"] * r["state"]
            t.update({x + "left.q": [a["heads"] * a["dim"], w], x + "left.k": [a["kv_heads"] * a["dim"], w], x + "left.v": [a["kv_heads"] * a["vdim"], w],
                      x + "left.o": [w, a["heads"] * a["vdim"]], x + "right.in": [2 * inner + 2 * gn + r["heads"], w], x + "right.conv": [inner + 2 * gn, r["conv"]],
                      x + "right.conv.b": [inner + 2 * gn], x + "right.dt_bias": [r["heads"]], x + "right.A_log": [r["heads"]], x + "right.D": [r["heads"]],
                      x + "right.norm": [inner], x + "right.o": [w, inner]})
        else:
            h, qk, vd = m["heads"], m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            t.update({x + "q": [qk, w], x + "q.conv": [qk, m["conv"]], x + "k": [qk, w], x + "k.conv": [qk, m["conv"]], x + "v": [vd, w],
                      x + "v.conv": [vd, m["conv"]], x + "b": [h, w], x + "a": [h, w], x + "dt_bias": [h], x + "A_log": [h], x + "norm": [m["vdim"]],
                      x + "g": [vd, w], x + "o": [w, vd]})
        f = layer["mlp"]["ff"]
        t.update({p + "mlp.gate": [f, w], p + "mlp.up": [f, w], p + "mlp.down": [w, f], p + "side.gate": [side, w], p + "side.proj": [w, side], p + "side.norm": [w]})
    t.update({"final.norm": [w], "head": [cfg["vocab"], w]})
    return t


def gugedra_decode_bytes(cfg: dict, pos: int) -> int:
    """Bytes one bf16 decode step at position pos has to move: every matrix once, the states read and written, the visible keys."""
    total = 2 * sum(int(np.prod(s)) for n, s in gugedra_shapes(cfg).items() if n not in ("embed", "side.embed")) + 2 * cfg["width"]
    for layer in cfg["layers"]:
        m = layer["mixer"]
        if layer["type"] == "parallel":
            a, r = m["left"], m["right"]
            total += 2 * min(pos + 1, a["mask"]["size"]) * a["kv_heads"] * (a["dim"] + a["vdim"]) + 8 * r["heads"] * r["state"] * r["vdim"]
        else:
            total += 8 * m["heads"] * m["dim"] * m["vdim"]
    return total


def gugedra_prefill_flops(cfg: dict, tokens: int) -> dict:
    """Operations of a prompt of `tokens` tokens: products with weights, attention inside the window, the recurrences."""
    skip = ("embed", "side.embed", "head")
    mm = sum(2 * tokens * int(np.prod(s)) for n, s in gugedra_shapes(cfg).items() if len(s) == 2 and n not in skip and not n.endswith(".conv"))
    attn = rec = 0
    for layer in cfg["layers"]:
        m = layer["mixer"]
        if layer["type"] == "parallel":
            a, r = m["left"], m["right"]
            w = min(a["mask"]["size"], tokens)
            attn += 2 * (w * (w + 1) // 2 + (tokens - w) * w) * a["heads"] * (a["dim"] + a["vdim"])
            rec += 5 * tokens * r["heads"] * r["state"] * r["vdim"]
        else:
            rec += 7 * tokens * m["heads"] * m["dim"] * m["vdim"]
    return {"matmul": mm, "attention": attn, "recurrence": rec}
