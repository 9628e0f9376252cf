"""Gugedra on the GPU against the float64 oracle (oracle/gugedra.py): the new operators alone, every layer alone, prompts, portions,
decoding, window, chunk and ring edges, states that last, and generation through the session."""

import json
import os
import pathlib
import subprocess
import sys

import numpy as np
import pytest

import brasa_b200 as B
from oracle import dunuzen as D
from oracle import gugedra as G

from dunuzen_cases import off, tokens
from gugedra_cases import CASES, attn, build, config, delta, parallel, ssm
from stack_helpers import bf16_array, follows, pad, portions

pytestmark = pytest.mark.gpu
ROOT = pathlib.Path(__file__).resolve().parent.parent
DTYPES = {"float32": 1e-4, "bfloat16": 8e-2}  # `off` of the logits of these peaked random models, as far as rounding allows (agree)
LAYER = {"float32": 3e-5, "bfloat16": 4e-2}


@pytest.fixture(scope="module")
def ctx():
    c = B.Context(0)
    yield c
    c.close()


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base, made = tmp_path_factory.mktemp("gugedra"), {}

    def get(name):
        if name not in made:
            cfg, w = build(name)
            D.write_model(base / name, cfg, w)
            made[name] = (base / name, cfg, w)
        return made[name]
    return get


_want = {}


def oracle(cfg, w, ids):
    key = (json.dumps(cfg), w["embed"].tobytes()[:64], ids.tobytes())
    if key not in _want:
        _want[key] = G.forward(cfg, w, ids)
    return _want[key]


_carried = {}


def agree(got, cfg, w, ids, dtype, rows=slice(None)):
    """Logits against the oracle's. In bfloat16 a peaked model carries rounding far at single positions: as far, three times over,
    as it carries the oracle's own; half of all positions stay within three times what half of the oracle's do."""
    want = oracle(cfg, w, ids)[0][rows]
    row = lambda a: np.sqrt(np.square((a - want) - (a - want).mean(-1, keepdims=True)).mean(-1)) / np.std(want, axis=-1)
    e = row(np.asarray(got, np.float64))
    if dtype == "float32":
        return e.max() <= DTYPES[dtype]
    key = (json.dumps(cfg), ids.tobytes())
    if key not in _carried:
        _carried[key] = G.forward(cfg, w, ids, D.bf16_round)[0]
    c = row(_carried[key][rows])
    return e.max() <= max(DTYPES[dtype], 3 * c.max()) and np.median(e) <= max(5e-3, 3 * np.median(c))


def load(ctx, path, dtype, ctx_len=512, max_tokens=512, rows=512):
    return B.Gugedra.load_in(ctx, path, dtype, ctx_len, max_tokens, rows)


# ---- operators -------------------------------------------------------------------------------------------------------------


@pytest.mark.parametrize("rows, n", [(1, 3), (5, 100), (3, 1001), (2, 2560), (2, 6000)])
@pytest.mark.parametrize("with_y, with_w, store", [(True, True, True), (False, True, False), (True, False, True), (True, True, False)])
def test_add_rms_norm(ctx, rows, n, with_y, with_w, store):
    rng = np.random.default_rng(n)
    x, y = [(rng.standard_normal((rows, n)) * s).astype(np.float32) for s in (3, 0.01)]
    wy, w = [rng.standard_normal(n).astype(np.float32) for _ in range(2)]
    bx, out = ctx.buffer_from(x), ctx.buffer(x.nbytes)
    cmd = ctx.command()
    B.Kernels(ctx).add_rms_norm(cmd, bx, ctx.buffer_from(y) if with_y else None, ctx.buffer_from(wy) if with_y else None, bx if store else None,
                                ctx.buffer_from(w) if with_w else None, out, rows, n, 1e-3)
    cmd.wait()
    x1 = x + G.rms_norm(y.astype(np.float64), wy, 1e-3) if with_y else x.astype(np.float64)
    want = G.rms_norm(x1, w, 1e-3) if with_w else x1
    assert np.abs(out.download(np.float32).reshape(rows, n) - want).max() <= 3e-6 * np.abs(want).max()
    assert np.abs(bx.download(np.float32).reshape(rows, n) - (x1 if store else x)).max() <= 2e-6 * np.abs(x1).max()


def interleaved(gate, up):
    """Alternating blocks of 32 rows, zero rows behind the last ones."""
    rows, cols = gate.shape
    n = (rows + 31) // 32 * 32
    out = np.zeros((n // 32, 2, 32, cols), gate.dtype)
    for i, m in enumerate((gate, up)):
        out[:, i] = np.concatenate([m, np.zeros((n - rows, cols), m.dtype)]).reshape(n // 32, 32, cols)
    return out.reshape(2 * n, cols)


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("n, rows, cols", [(2, 7, 40), (130, 70, 72), (257, 512, 136), (900, 1000, 64)])
def test_linear_epilogues(ctx, n, rows, cols, f32):
    """silu(gate) up out of interleaved rows; gelu times a gathered row; a softcap; all in one launch."""
    rng, K, ids_n = np.random.default_rng(rows), B.Kernels(ctx), 19
    x = D.bf16_round(rng.standard_normal((n, cols)))
    gate, up, ge, cap = [D.bf16_round(2 * rng.standard_normal((rows, cols)) / np.sqrt(cols)) for _ in range(4)]
    table, ids = D.bf16_round(rng.standard_normal((ids_n, rows + 3))), rng.integers(0, ids_n, n).astype(np.uint32)
    ld, xb = (cols + 7) // 8 * 8, lambda a: ctx.buffer_from(a if f32 else D.bf16_bits(a))
    bx, wb = xb(pad(x, ld)), lambda m: ctx.buffer_from(D.bf16_bits(pad(m, ld)))
    glu = interleaved(gate, up)
    y = [ctx.buffer(n * r * 4) for r in (len(glu) // 2, rows, rows)]
    cmd = ctx.command()
    K.linear(cmd, [K.linear_problem(wb(glu), bx, y[0], len(glu), cols, n, ld, ld, len(glu) // 2, act=K.ACT_SWIGLU),
                   K.linear_problem(wb(ge), bx, y[1], rows, cols, n, ld, ld, rows, act=K.ACT_GELU_TANH, mul=ctx.buffer_from(D.bf16_bits(table)),
                                    mul_ids=ctx.buffer_from(ids), ldm=rows + 3, mul_rows=ids_n),
                   K.linear_problem(wb(cap), bx, y[2], rows, cols, n, ld, ld, rows, scale=3.0, cap=2.5)], f32)
    cmd.wait()
    x = x.astype(np.float64)
    want = [D.silu(x @ gate.T) * (x @ up.T), G.gelu_tanh(x @ ge.T) * table[ids][:, :rows], G.softcap(3.0 * (x @ cap.T), 2.5)]
    for b, r in zip(y, want):
        got = b.download(np.float32).reshape(n, -1)
        assert np.abs(got[:, :rows] - r).max() <= 1e-5 * np.abs(r).max() and not got[:, rows:].any()


WINDOWS = [  # heads, kv_heads, dim, vdim, rot_dims, window, pos0, tokens, ring, softcap
    (4, 2, 32, 32, 32, 5, 0, 40, 0, 8.0), (6, 2, 64, 64, 16, 128, 0, 300, 384, 30.0), (3, 1, 96, 128, 24, 129, 200, 131, 384, 5.0), (2, 2, 128, 64, 128, 1000, 0, 257, 0, 0.0),
    (8, 1, 192, 128, 64, 127, 1000, 2, 128, 50.0), (2, 1, 16, 72, 6, 1, 3, 130, 256, 12.0), (1, 1, 200, 200, 10, 33, 77, 65, 128, 20.0), (4, 4, 64, 128, 32, 256, 255, 256, 512, 0.0),
    (2, 1, 64, 64, 64, 200, 900, 150, 384, 100.0), (5, 5, 40, 24, 20, 64, 640, 64, 128, 64.0), (2, 1, 128, 128, 48, 300, 1500, 400, 768, 30.0)]


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("heads, kv, dim, vdim, rot, window, pos0, n, ring, cap", WINDOWS)
def test_window_attention_of_shared_heads(ctx, heads, kv, dim, vdim, rot, window, pos0, n, ring, cap, f32):
    """Keys one behind the other or in a ring; two queries' last visible key and the one before it both answer them strongly."""
    rng = np.random.default_rng(dim + window)
    first, last, scale, share = max(0, pos0 + 1 - window), pos0 + n, dim ** -0.5, heads // kv
    key0 = first // 128 * 128 if ring else first
    q = (2.0 * rng.standard_normal((n, heads, dim))).astype(np.float32)
    pos, kp = np.arange(pos0, last), np.arange(key0, last)
    qr = D.rope_half(q.astype(np.float64), pos, rot, 700.0)
    k, v = (D.bf16_round(rng.standard_normal((last - key0, kv, s))) for s in (dim, vdim))
    for t in (0, n // 2):
        for j in (pos0 + t - window + 1, pos0 + t - window):
            if key0 <= j < last:
                to = qr[t, ::share]
                k[j - key0] = D.bf16_round(3.0 * to / np.linalg.norm(to, axis=-1, keepdims=True) * np.sqrt(dim))

    def placed(a):  # in the ring, other rows: large but finite
        if not ring:
            return a
        r = np.full((ring,) + a.shape[1:], 3e4, a.dtype)
        for p in range(max(first, last - ring), last):
            r[p % ring] = a[p - key0]
        return r
    dev = (lambda a: ctx.buffer_from(np.ascontiguousarray(a, np.float32))) if f32 else (lambda a: ctx.buffer_from(D.bf16_bits(a)))
    out, cmd = ctx.buffer(n * heads * vdim * (4 if f32 else 2)), ctx.command()
    B.Kernels(ctx).window_attention(cmd, ctx.buffer_from(q), dev(placed(k)), dev(placed(v)), None, B.RopeTable(ctx, 700.0, rot, last), None, out, n, heads, dim, 0, vdim, pos0,
                                    key0, window, scale, f32, kv, ring, cap, 0.75)
    cmd.wait()
    got = (out.download(np.float32) if f32 else bf16_array(out.download(np.uint16))).reshape(n, heads, vdim)
    seen = (pos[:, None] - kp[None, :] >= 0) & (pos[:, None] - kp[None, :] < window)
    want = np.zeros((n, heads, vdim))
    for h in range(heads):
        s = qr[:, h] @ k[:, h // share].T.astype(np.float64) * scale
        want[:, h] = 0.75 * D.softmax_rows(G.softcap(s, cap) if cap else s, seen) @ v[:, h // share].astype(np.float64)
    assert np.abs(got - want).max() <= (2e-5 if f32 else 5e-2) * np.abs(want).max()
    assert np.sqrt(((got - want) ** 2).mean()) <= (4e-6 if f32 else 6e-3) * np.abs(want).max()


# ---- layers ----------------------------------------------------------------------------------------------------------------


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CASES)
def test_each_layer_alone(ctx, folders, name, dtype):
    """A layer on a random residual stream: as one run, token by token, in short portions, and cut at and beside the chunks' edges."""
    path, cfg, w = folders(name)
    m = load(ctx, path, dtype)
    n, dim = 150, cfg["token_side"]["dim"]
    x, ids = np.random.default_rng(5).standard_normal((n, cfg["width"])).astype(np.float32) * 2, tokens(cfg, 150, 6)
    for i, layer in enumerate(cfg["layers"]):
        want = G.layer(x.astype(np.float64), w["side.embed"][ids][:, i * dim:(i + 1) * dim].astype(np.float64), cfg, layer,
                       lambda s: w[f"l{i}." + s].astype(np.float64)) - x

        def cut(sizes):
            out, at, k = [], 0, 0
            while at < n:
                c = min(sizes[k % len(sizes)], n - at)
                out.append(m.run_layers(x[at:at + c], at, range(i, i + 1), ids[at:at + c]).reshape(c, -1))
                at, k = at + c, k + 1
            return np.concatenate(out) - x
        for sizes in ([n], [1], [2], [5, 1], [64, 1, 63, 16], [65], [100, 1, 1, 7]):
            got = cut(sizes)
            err = np.sqrt(((got - want) ** 2).mean()) / np.sqrt((want ** 2).mean())
            assert err <= LAYER[dtype], (i, layer["type"], sizes, err)
    with pytest.raises(B.BrasaError):  # its layers read the tokens too
        m.run_layers(x[:2], 0, range(0, 1))
    m.free()


# ---- whole models ----------------------------------------------------------------------------------------------------------


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CASES)
def test_prompts_portions_and_decoding(ctx, folders, name, dtype):
    path, cfg, w = folders(name)
    ids = tokens(cfg, 210)
    m = load(ctx, path, dtype)
    whole = portions(m, ids, [210])
    assert agree(whole, cfg, w, ids, dtype)
    assert np.array_equal(whole, portions(m, ids, [210]))  # what an earlier sequence left behind changes nothing
    for sizes in ([2], [1], [3, 64, 2, 19], [100, 1, 1, 1], [128]):
        assert agree(portions(m, ids, sizes), cfg, w, ids, dtype), sizes
    m.free()


@pytest.mark.parametrize("width", [4100, 6004])
def test_wide_stream(ctx, tmp_path, width):
    """A residual stream wider than the single-token product keeps in registers, and than a norm's block does."""
    cfg = config(width, 40, [(parallel(attn(2, 1, 16, 8, 9, 8), ssm(2, 8, 16, 1, 2, 3)), 24), (delta(1, 1, 8, 8, 2), None)])
    w = G.random_weights(cfg, 0)
    D.write_model(tmp_path, cfg, w)
    ids = tokens(cfg, 24)
    for dtype in DTYPES:
        m = load(ctx, tmp_path, dtype, ctx_len=32, max_tokens=32, rows=32)
        for sizes in ([24], [1], [10, 1, 1]):
            assert agree(portions(m, ids, sizes), cfg, w, ids, dtype), (dtype, sizes)
        m.free()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["ragged", "ones"])
def test_first_tokens(ctx, folders, name, dtype):
    """Sequences shorter than the convolutions and the windows, one after the other in the same state."""
    path, cfg, w = folders(name)
    m = load(ctx, path, dtype, max_tokens=64, rows=64)
    for n in (1, 2, 3, 4, 5, 9):
        ids = tokens(cfg, n, seed=n)
        assert agree(portions(m, ids, [n]), cfg, w, ids, dtype)
        assert agree(portions(m, ids, [1]), cfg, w, ids, dtype)
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["ragged", "tiles", "ones"])
def test_ring_turns_over(ctx, folders, name, dtype):
    """Runs so short that the rings of keys and values turn over again and again, in prompts and in long decoding."""
    path, cfg, w = folders(name)
    ids = tokens(cfg, 900, seed=9)
    m = load(ctx, path, dtype, ctx_len=900, max_tokens=48, rows=48)
    assert agree(portions(m, ids, [48]), cfg, w, ids, dtype)
    assert agree(portions(m, ids, [31, 2, 48]), cfg, w, ids, dtype)
    first = portions(m, ids[:300], [48])
    decoded = np.concatenate([m.feed(ids[t:t + 1], t, [0]) for t in range(300, 900)])
    assert agree(np.concatenate([first, decoded]), cfg, w, ids, dtype)
    m.free()


def edge_model(window, mark, d=24, width=64, vocab=48):
    """One parallel layer whose heads look for one token: the query of every token answers only the key of token `mark`, far above
    all others, so that the output tells whether that token is in sight. The other side is held small."""
    cfg = config(width, vocab, [(parallel(attn(4, 2, d, 16, window, 8, scale=1.0, softcap=30.0), ssm(2, 8, 8, 1, 1, 2), 1.0, 0.02), None)], side=4)
    w = G.random_weights(cfg, 11)
    w["l0.norm1"][:], w["l0.side.norm"][:] = 1.0, 0.05
    emb = np.zeros((vocab, width))
    emb[:, 8:] = 0.5 * np.random.default_rng(0).standard_normal((vocab, width - 8))
    emb[:, 0], emb[:, 1] = 4.0, -4.0         # every token carries the query direction ..
    emb[mark, 2], emb[mark, 3] = 9.0, -9.0   # .. and the marked one the key direction
    w["embed"] = D.bf16_round(emb)
    q, k = np.zeros((4 * d, width)), np.zeros((2 * d, width))
    q[d - 1::d, 0] = 3.0                     # the heads' last entries, which are not rotated
    k[d - 1::d, 2] = 4.0
    w["l0.mix.left.q"], w["l0.mix.left.k"] = D.bf16_round(q), D.bf16_round(k)
    return cfg, w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [2, 16, 63, 64, 65, 128, 150])
def test_window_edge_shows(ctx, tmp_path, window, dtype):
    """The marked token at position 40 is seen up to position 40 + window - 1 and not one further."""
    mark, at = 7, 40
    cfg, w = edge_model(window, mark)
    D.write_model(tmp_path, cfg, w)
    n = at + window + 30
    ids = tokens(cfg, n, seed=window)
    ids[ids == mark] = mark + 1
    ids[at] = mark
    want, after = oracle(cfg, w, ids)
    clean = ids.copy()
    clean[at] = mark + 1
    plain = G.forward(cfg, w, clean)[1]
    last, next_ = at + window - 1, at + window
    # the test can tell: the edge's inside moves a lot, its outside hardly
    assert np.abs(after[0, last] - plain[0, last]).max() > 0.3 > 6 * np.abs(after[0, next_] - plain[0, next_]).max()
    m = load(ctx, tmp_path, dtype, ctx_len=n, max_tokens=64, rows=64)
    for sizes in ([64], [37, 1, 2], [1]):
        got = portions(m, ids, sizes)
        assert agree(got, cfg, w, ids, dtype), sizes
        assert agree(got[last:next_ + 1], cfg, w, ids, dtype, slice(last, next_ + 1)), sizes
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("side", ["delta", "state space"])
def test_states_remember(ctx, tmp_path, side, dtype):
    """Decays close to one: what the first tokens wrote still decides the last ones' logits, across portions and decoding."""
    if side == "delta":
        cfg = config(64, 60, [(delta(4, 2, 24, 16, 4), None)])
        x = "l0.mix."
    else:
        cfg = config(64, 60, [(parallel(attn(2, 1, 8, 8, 2, 4), ssm(4, 24, 40, 2, 2, 4), 0.1, 1.0), None)])
        x = "l0.mix.right."
    w = G.random_weights(cfg, 2)
    w[x + "A_log"][:], w[x + "dt_bias"][:] = -7.0, -1.0
    D.write_model(tmp_path, cfg, w)
    ids = tokens(cfg, 200, seed=4)
    want, _ = oracle(cfg, w, ids)
    other = ids.copy()
    other[:3] = (other[:3] + 1) % 60
    assert off(G.forward(cfg, w, other)[0][-1:], want[-1:]) > 10 * DTYPES["float32"]  # the first tokens do matter at the end
    m = load(ctx, tmp_path, dtype)
    for sizes in ([200], [2], [77, 1], [1]):
        assert agree(portions(m, ids, sizes), cfg, w, ids, dtype), sizes
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
def test_states_forget(ctx, tmp_path, dtype):
    """Decays down to nothing inside a chunk."""
    cfg = config(64, 60, [(parallel(attn(2, 1, 8, 8, 2, 4), ssm(4, 24, 40, 2, 2, 4), 0.1, 1.0), None), (delta(4, 2, 24, 16, 4), 32)])
    w = G.random_weights(cfg, 2)
    for x in ("l0.mix.right.", "l1.mix."):
        w[x + "A_log"][:], w[x + "dt_bias"][:] = [3.0, 5.0, -2.0, 2.0], [2.0, 6.0, 0.0, -1.0]
    D.write_model(tmp_path, cfg, w)
    ids = tokens(cfg, 150, seed=4)
    m = load(ctx, tmp_path, dtype)
    for sizes in ([150], [70, 1], [1]):
        assert agree(portions(m, ids, sizes), cfg, w, ids, dtype), sizes
    m.free()


def test_constants_are_read(ctx, tmp_path):
    """Every constant of the configuration changes the result the way it changes the oracle's."""
    base, w = build("ragged")
    ids = tokens(base, 60)
    ref, _ = G.forward(base, w, ids)
    left, right = (lambda c: c["layers"][1]["mixer"]["left"]), (lambda c: c["layers"][1]["mixer"]["right"])
    changes = [lambda c: c.update(logit_softcap=3.0), lambda c: c["norm"].update(eps=0.3), lambda c: left(c)["mask"].update(size=7), lambda c: left(c)["rot"].update(base=3.0),
               lambda c: left(c)["rot"].update(dims=4), lambda c: left(c).update(scale=0.05), lambda c: left(c).update(softcap=1.5), lambda c: right(c).update(norm_groups=6),
               lambda c: c["layers"][1]["mixer"].update(left_scale=0.1), lambda c: c["layers"][2]["mixer"].update(right_scale=2.0),
               lambda c: c["layers"][2]["mixer"]["left"]["mask"].update(size=51), lambda c: c["layers"][3].update(mlp=None)]
    for i, change in enumerate(changes):
        cfg = json.loads(json.dumps(base))
        change(cfg)
        D.write_model(tmp_path / str(i), cfg, w)
        want, _ = G.forward(cfg, w, ids)
        assert np.abs(want - ref).max() > 1e-3 or i == len(changes) - 1
        m = load(ctx, tmp_path / str(i), "float32")
        for sizes in ([60], [1]):
            assert np.abs(portions(m, ids, sizes) - want).max() <= 2e-4 * np.abs(want).max(), (i, sizes)
        m.free()


# ---- state bookkeeping, memory, generation ---------------------------------------------------------------------------------


def test_state_goes_forward_only(ctx, folders):
    path, cfg, w = folders("tiles")
    m = load(ctx, path, "float32", rows=4)
    ids = tokens(cfg, 30)
    m.feed(ids[:20], 0, [19])
    for bad in (5, 19, 21):
        with pytest.raises(B.BrasaError) as e:
            m.feed(ids[20:25], bad, [0])
        assert e.value.code == B.EINVAL
    good = m.feed(ids[20:25], 20, [4])  # a refused call leaves the state as it was
    want, _ = oracle(cfg, w, ids)
    assert off(good, want[24:25]) <= DTYPES["float32"]
    assert off(m.feed(ids[:3], 0, [2]), want[2:3]) <= DTYPES["float32"]  # position 0 starts over
    with pytest.raises(B.BrasaError):
        B.Batch(m, 2, 8, 64)
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CASES)
def test_plan_is_what_is_allocated(ctx, folders, name, dtype):
    path, _, _ = folders(name)
    m = load(ctx, path, dtype, ctx_len=300, max_tokens=70, rows=9)
    _, plan, _ = B.planner.check_path(ctx, path, m.limits)
    assert {k: plan[k] for k in ("weights", "kv", "workspace")} == m.allocated()
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["ragged", "tiles"])
def test_greedy_generation(ctx, folders, name, dtype):
    path, cfg, w = folders(name)
    tol = 4 * DTYPES[dtype]
    s = B.Session(ctx, path, B.Limits(ctx=400, max_tokens=32, kv=B.Gugedra.kv_type(dtype)))
    prompt = tokens(cfg, 75, seed=3)
    ids, st = s.generate(prompt, 40)
    assert len(ids) == 40 and st.stop == "MaxTokens" and st.reused_tokens == 0
    follows(G.forward, cfg, w, prompt, ids, tol)
    # the conversation goes on: all of it is reused; then a prompt that branches off: none of it
    more = np.concatenate([prompt, ids, tokens(cfg, 11, seed=8)])
    ids2, st2 = s.generate(more, 10)
    assert st2.reused_tokens == 115
    follows(G.forward, cfg, w, more, ids2, tol)
    branch = np.concatenate([prompt[:50], tokens(cfg, 9, seed=2)])
    ids3, st3 = s.generate(branch, 10)
    assert st3.reused_tokens == 0
    follows(G.forward, cfg, w, branch, ids3, tol)
    # the device-resident loop through the model
    s.model.forward(prompt[:32], 0)
    s.model.forward(prompt[32:64], 32)
    logits, _ = s.model.forward(prompt[64:], 64)
    first = int(np.argmax(logits[0]))
    dev, _ = s.model.decode_greedy(first, 75, 12)
    assert [first] + list(dev[:11]) == list(ids[:12])
    s.free()


def test_sampled_generation(ctx, folders):
    path, cfg, w = folders("tiles")
    params = B.SamplingParams(temperature=0.8, top_k=20, top_p=0.9, seed=5)
    s = B.Session(ctx, path, B.Limits(ctx=200, max_tokens=64, kv=B.KvType.F32))
    prompt = tokens(cfg, 30)
    ids, _ = s.generate(prompt, 25, params)
    s.reset()
    again, _ = s.generate(prompt, 25, params)
    assert list(ids) == list(again) and len(set(ids)) > 3
    lg, _ = G.forward(cfg, w, np.concatenate([prompt, ids]))
    for i, t in enumerate(ids):  # every draw is among the oracle's twenty best
        assert (lg[29 + i] > lg[29 + i][t] + 1e-3).sum() < 20
    s.free()


def test_graph_and_plain_steps_agree(ctx, folders):
    path, cfg, _ = folders("tiles")
    code = ("import sys, numpy as np; sys.path.insert(0, sys.argv[1]); import brasa_b200 as B; c = B.Context(0); "
            "m = B.Gugedra.load_in(c, sys.argv[2], 'bfloat16', 200, 64); l, _ = m.forward(np.arange(50), 0); "
            "print(list(map(int, m.decode_greedy(int(np.argmax(l[0])), 50, 30)[0])))")
    outs = []
    for env in ({}, {"BRASA_GRAPH": "0"}, {"BRASA_PDL": "0"}):
        r = subprocess.run([sys.executable, "-c", code, str(ROOT), str(path)], capture_output=True, text=True, env={**os.environ, **env}, timeout=120)
        assert r.returncode == 0, r.stderr
        outs.append(r.stdout)
    assert outs[0] == outs[1] == outs[2]


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_runner_program(ctx, folders, tmp_path, dtype):
    path, cfg, w = folders("ragged")
    ids = tokens(cfg, 40)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": ids[:30].tolist(), "want": [0, 29, 7]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": ids[30:31].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": ids[31:].tolist(), "want": [8]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": ids[:2].tolist(), "want": [1]}], "end": ["y"]}]
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(path), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "40"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    for step, rows in ((0, [0, 29, 7]), (2, [39]), (3, [1])):
        got = np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(len(rows), -1)
        assert agree(got, cfg, w, ids, dtype, rows)
    assert not (tmp_path / "1.f32").exists()


def test_command_line_generates(ctx, folders):
    path, cfg, w = folders("tiles")
    prompt = tokens(cfg, 20)
    r = subprocess.run([sys.executable, "-m", "brasa_b200", "generate", str(path), "--prompt", ",".join(map(str, prompt)), "--max-new", "8", "--dtype", "float32"],
                       capture_output=True, text=True, cwd=ROOT, timeout=120)
    assert r.returncode == 0, r.stderr
    ids = np.array([int(t) for t in r.stdout.split()])
    assert len(ids) == 8
    follows(G.forward, cfg, w, prompt, ids, 1e-3)
