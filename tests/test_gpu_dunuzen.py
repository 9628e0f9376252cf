"""Dunuzen on the GPU against the float64 oracle (oracle/dunuzen.py): the new operators alone, every layer alone, prompts, portions,
decoding, the end of windows and the turn of the ring, and generation through the session."""

import json
import os
import pathlib
import subprocess
import sys

import numpy as np
import pytest

import brasa_b200 as B
from oracle import dunuzen as D

from dunuzen_cases import CASES, LA, build, config, delta, latent, off, tokens
from stack_helpers import follows, pad, portions

pytestmark = pytest.mark.gpu
ROOT = pathlib.Path(__file__).resolve().parent.parent
DTYPES = {"float32": 1e-4, "bfloat16": 6e-2}  # `off` of the logits of these peaked random models
LAYER = {"float32": 3e-5, "bfloat16": 4e-2}


@pytest.fixture(scope="module")
def ctx():
    c = B.Context(0)
    yield c
    c.close()


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base, made = tmp_path_factory.mktemp("dunuzen"), {}

    def get(name, **kw):
        key = (name, tuple(sorted(kw.items())))
        if key not in made:
            cfg, w = build(name, **kw)
            path = base / f"{name}{len(made)}"
            D.write_model(path, cfg, w)
            made[key] = (path, cfg, w)
        return made[key]
    return get


_want = {}


def oracle(cfg, w, ids):
    key = (json.dumps(cfg), w["embed"].tobytes()[:64], ids.tobytes())
    if key not in _want:
        _want[key] = D.forward(cfg, w, ids)
    return _want[key]


def load(ctx, path, dtype, ctx_len=512, max_tokens=512, rows=512):
    return B.Dunuzen.load_in(ctx, path, dtype, ctx_len, max_tokens, rows)


# ---- operators -------------------------------------------------------------------------------------------------------------


@pytest.mark.parametrize("rows, n", [(1, 4), (5, 100), (3, 1000), (2, 2560)])
def test_layer_norm(ctx, rows, n):
    rng = np.random.default_rng(n)
    x, w, b = (rng.standard_normal((rows, n)) * 3 + 5).astype(np.float32), rng.standard_normal(n).astype(np.float32), rng.standard_normal(n).astype(np.float32)
    out = ctx.buffer(x.nbytes)
    cmd = ctx.command()
    B.Kernels(ctx).layer_norm(cmd, ctx.buffer_from(x), ctx.buffer_from(w), ctx.buffer_from(b), out, rows, n, 1e-3)
    cmd.wait()
    want = D.layer_norm(x.astype(np.float64), w, b, 1e-3)
    assert np.abs(out.download(np.float32).reshape(rows, n) - want).max() <= 2e-5 * np.abs(want).max()


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("tokens_n, shapes", [
    (2, [(7, 40, 0)]), (130, [(65, 72, 0), (300, 72, 24), (1, 8, 0)]), (257, [(512, 512, 136)]), (700, [(1300, 320, 64), (40, 64, 0)]),
    (2000, [(2600, 192, 0)]), (3, [(5000, 1000, 0)])])
def test_linear_group(ctx, tokens_n, shapes, f32):
    """Every tile width, ragged edges, one and two segments, bias, squared relu, scale, residual in place, both output types."""
    rng = np.random.default_rng(tokens_n)
    K, up8, probs, wants, bufs = B.Kernels(ctx), lambda v: (v + 7) // 8 * 8, [], [], []
    for i, (rows, cols, cols2) in enumerate(shapes):
        seg = []
        want = 0.0
        for c in (cols, cols2):
            if not c:
                continue
            w, x = D.bf16_round(rng.standard_normal((rows, c)) / np.sqrt(c)), D.bf16_round(rng.standard_normal((tokens_n, c)))
            want = want + x.astype(np.float64) @ w.T.astype(np.float64)
            xb = pad(x, up8(c) + 8)
            seg.append((ctx.buffer_from(D.bf16_bits(pad(w, up8(c)))), ctx.buffer_from(xb if f32 else D.bf16_bits(xb)), c, up8(c), up8(c) + 8))
        bias = rng.standard_normal(rows).astype(np.float32)
        relu2, in_place = i % 2 == 1, i % 2 == 0
        want = want + bias
        if relu2:
            want = np.maximum(want, 0) ** 2
        want = want * 1.5
        ldy = up8(rows) if i else rows
        res = rng.standard_normal((tokens_n, ldy)).astype(np.float32)
        y = ctx.buffer_from(res) if in_place else ctx.buffer(tokens_n * ldy * 2)
        if in_place:
            want = want + res[:, :rows]
        (w0, x0, c0, lw0, lx0), second = seg[0], seg[1] if len(seg) > 1 else (None, None, 0, 0, 0)
        probs.append(K.linear_problem(w0, x0, y, rows, c0, tokens_n, lw0, lx0, ldy, second[0], second[1], second[2], second[3], second[4], ctx.buffer_from(bias),
                                      y if in_place else None, not in_place, relu2, 1.5))
        bufs.append((y, ldy, in_place, seg))
        wants.append(want)
    cmd = ctx.command()
    K.linear(cmd, probs, f32)
    cmd.wait()
    for (y, ldy, in_place, _), want in zip(bufs, wants):
        if in_place:
            got = y.download(np.float32).reshape(tokens_n, ldy)
        else:
            got = (y.download(np.uint16).astype(np.uint32) << 16).view(np.float32).reshape(tokens_n, ldy)
        tol = (2e-5 if in_place else 8e-3) * np.abs(want).max()
        assert np.abs(got[:, :want.shape[1]] - want).max() <= tol


WINDOWS = [  # heads, dim, rot, vdim, window, pos0, tokens
    (2, 32, 16, 32, 5, 0, 40), (3, 64, 8, 64, 128, 0, 300), (1, 96, 32, 128, 129, 200, 131), (2, 128, 64, 128, 1000, 0, 257), (1, 192, 64, 64, 127, 1000, 2),
    (2, 16, 8, 72, 1, 3, 130), (1, 136, 16, 200, 33, 77, 65), (2, 64, 24, 128, 256, 255, 256)]


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("heads, dim, rot, vdim, window, pos0, n", WINDOWS)
def test_window_attention(ctx, heads, dim, rot, vdim, window, pos0, n, f32):
    """Scores peaked by scaled queries; then one key per query made to stand out at exactly the last visible place and one just
    behind it, which must not be seen."""
    rng = np.random.default_rng(dim + window)
    key0 = max(0, pos0 + 1 - window)
    keys, last = pos0 + n - key0, pos0 + n
    q, gate = (2.0 * rng.standard_normal((n, heads, dim + rot))).astype(np.float32), rng.standard_normal((n, heads)).astype(np.float32)
    k, v, kr = (D.bf16_round(rng.standard_normal(s)) for s in ((keys, heads, dim), (keys, heads, vdim), (keys, rot)))
    pos = np.arange(pos0, last)
    # the first query's edge: its last visible key and the one before it both answer it strongly
    for j in (pos0 - window + 1, pos0 - window):
        if 0 <= j - key0:
            k[j - key0] = D.bf16_round(3.0 * q[0, :, :dim] / np.linalg.norm(q[0, :, :dim], axis=-1, keepdims=True) * np.sqrt(dim))
    mid = n // 2
    for j in (pos0 + mid - window + 1, pos0 + mid - window):
        if 0 <= j - key0 < keys:
            k[j - key0] = D.bf16_round(3.0 * q[mid, :, :dim] / np.linalg.norm(q[mid, :, :dim], axis=-1, keepdims=True) * np.sqrt(dim))
    table, scale = B.RopeTable(ctx, 700.0, rot, last), (dim + rot) ** -0.5
    dev = (lambda a: ctx.buffer_from(np.ascontiguousarray(a, np.float32))) if f32 else (lambda a: ctx.buffer_from(D.bf16_bits(a)))
    out = ctx.buffer(n * heads * vdim * (4 if f32 else 2))
    cmd = ctx.command()
    B.Kernels(ctx).window_attention(cmd, ctx.buffer_from(q), dev(k), dev(v), dev(kr), table, ctx.buffer_from(gate), out, n, heads, dim, rot, vdim, pos0, key0, window,
                                    scale, f32)
    cmd.wait()
    got = (out.download(np.float32) if f32 else (out.download(np.uint16).astype(np.uint32) << 16).view(np.float32)).reshape(n, heads, vdim)
    qr = D.rope_half(q[..., dim:].astype(np.float64), pos, rot, 700.0)
    kp = np.arange(key0, last)
    seen = (pos[:, None] - kp[None, :] >= 0) & (pos[:, None] - kp[None, :] < window)
    want = np.zeros((n, heads, vdim))
    for h in range(heads):
        s = (q[:, h, :dim].astype(np.float64) @ k[:, h].T.astype(np.float64) + qr[:, h] @ kr.T.astype(np.float64)) * scale
        want[:, h] = D.softmax_rows(s, seen) @ v[:, h].astype(np.float64) * D.sigmoid(gate[:, h:h + 1].astype(np.float64))
    assert np.abs(got - want).max() <= (2e-5 if f32 else 5e-2) * np.abs(want).max()
    assert np.sqrt(((got - want) ** 2).mean()) <= (4e-6 if f32 else 6e-3) * np.abs(want).max()


# ---- layers ----------------------------------------------------------------------------------------------------------------


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CASES)
def test_each_layer_alone(ctx, folders, name, dtype):
    """A layer on a random residual stream: as one run, token by token, and in portions of two and five."""
    path, cfg, w = folders(name)
    m = load(ctx, path, dtype)
    n = 61
    x = np.random.default_rng(5).standard_normal((n, cfg["width"])).astype(np.float32) * 2
    for i, layer in enumerate(cfg["layers"]):
        f = lambda s: w[f"l{i}." + s].astype(np.float64)
        eps = cfg["norm"]["eps"]
        x64 = x.astype(np.float64)
        want = D.MIXERS[layer["type"]](D.layer_norm(x64, f("norm1"), f("norm1.b"), eps), lambda s: f("mix." + s), layer["mixer"], eps)
        if layer["mlp"]:
            want = want + D.feed_forward(D.layer_norm(x64, f("norm2"), f("norm2.b"), eps), lambda s: f("mlp." + s))

        def cut(sizes):
            out, at, k = [], 0, 0
            while at < n:
                c = min(sizes[k % len(sizes)], n - at)
                out.append(m.run_layers(x[at:at + c], at, range(i, i + 1)).reshape(c, -1))
                at, k = at + c, k + 1
            return np.concatenate(out) - x
        for sizes in ([n], [1], [2], [5, 1], [40, 1, 1, 7]):
            got = cut(sizes)
            err = np.sqrt(((got - want) ** 2).mean()) / np.sqrt((want ** 2).mean())
            assert err <= LAYER[dtype], (i, layer["type"], sizes, err)
    m.free()


# ---- whole models ----------------------------------------------------------------------------------------------------------


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CASES)
def test_prompts_portions_and_decoding(ctx, folders, name, dtype):
    path, cfg, w = folders(name)
    ids = tokens(cfg, 210)
    want, _ = oracle(cfg, w, ids)
    m = load(ctx, path, dtype)
    whole = portions(m, ids, [210])
    assert off(whole, want) <= DTYPES[dtype]
    assert np.array_equal(whole, portions(m, ids, [210]))  # what an earlier sequence left behind changes nothing
    for sizes in ([2], [1], [3, 64, 2, 19], [100, 1, 1, 1], [128]):
        assert off(portions(m, ids, sizes), want) <= DTYPES[dtype], sizes
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(ctx, folders, dtype):
    """Sequences shorter than the convolution and the windows, one after the other in the same state."""
    path, cfg, w = folders("ragged")
    m = load(ctx, path, dtype, max_tokens=64, rows=64)
    for n in (1, 2, 3, 4, 5, 9):
        ids = tokens(cfg, n, seed=n)
        want, _ = oracle(cfg, w, ids)
        assert off(portions(m, ids, [n]), want) <= DTYPES[dtype]
        assert off(portions(m, ids, [1]), want) <= DTYPES[dtype]
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["ragged", "tiles", "ones"])
def test_ring_turns_over(ctx, folders, name, dtype):
    """Runs so short that the ring of latent rows turns over again and again, in prompts and in long decoding."""
    path, cfg, w = folders(name)
    ids = tokens(cfg, 700, seed=9)
    want, _ = oracle(cfg, w, ids)
    m = load(ctx, path, dtype, ctx_len=700, max_tokens=48, rows=48)
    assert off(portions(m, ids, [48]), want) <= DTYPES[dtype]
    assert off(portions(m, ids, [31, 2, 48]), want) <= DTYPES[dtype]
    first = portions(m, ids[:300], [48])
    decoded = np.concatenate([m.feed(ids[t:t + 1], t, [0]) for t in range(300, 700)])
    assert off(np.concatenate([first, decoded]), want) <= DTYPES[dtype]
    m.free()


def edge_model(window, mark, d=16, width=64, vocab=48):
    """One latent layer whose heads look for one token: the query of every token answers only the key of token `mark`, far above
    all others, so that the output tells whether that token is in sight."""
    cfg = config(width, vocab, [(LA, latent(2, d, 8, 16, 24, window, scale=1.0), None)])
    w = D.random_weights(cfg, 11)
    w["l0.norm1"][:], w["l0.norm1.b"][:] = 1.0, 0.0
    emb = np.zeros((vocab, width))
    emb[:, 8:] = 0.5 * np.random.default_rng(0).standard_normal((vocab, width - 8))
    emb[:, 0], emb[:, 1] = 4.0, -4.0         # every token carries the query direction ..
    emb[mark, 2], emb[mark, 3] = 9.0, -9.0   # .. and the marked one the key direction
    w["embed"] = D.bf16_round(emb)
    q = np.zeros((2 * (d + 8), width))
    q[[0, d + 8], 0] = 4.0
    down = 0.2 * w["l0.mix.dkv"]
    down[0] = 0.0
    down[0, 2] = 8.0
    uk = np.zeros((2 * d, 24))
    uk[[0, d], 0] = 1.0
    w["l0.mix.q"], w["l0.mix.dkv"], w["l0.mix.uk"] = D.bf16_round(q), D.bf16_round(down), D.bf16_round(uk)
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
    plain = D.forward(cfg, w, clean)[1]
    last, next_ = at + window - 1, at + window
    # the test can tell: the edge's inside moves a lot, its outside not at all
    assert np.abs(after[0, last] - plain[0, last]).max() > 0.1 and np.allclose(after[0, next_], plain[0, next_])
    m = load(ctx, tmp_path, dtype, ctx_len=n, max_tokens=64, rows=64)
    for sizes in ([64], [37, 1, 2], [1]):
        got = portions(m, ids, sizes)
        assert off(got, want) <= DTYPES[dtype], sizes
        assert off(got[last:next_ + 1], want[last:next_ + 1]) <= DTYPES[dtype], sizes
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_state_remembers(ctx, tmp_path, dtype):
    """Decays close to one: what the first tokens wrote still decides the last ones' logits, across portions and decoding."""
    cfg = config(64, 60, [("channel_delta", delta(4, 2, 24, 16, 4), 64)])
    w = D.random_weights(cfg, 2)
    w["l0.mix.A_log"][:], w["l0.mix.dt_bias"][:] = -6.0, -4.0
    D.write_model(tmp_path, cfg, w)
    ids = tokens(cfg, 200, seed=4)
    want, _ = oracle(cfg, w, ids)
    other = ids.copy()
    other[:3] = (other[:3] + 1) % 60
    assert off(D.forward(cfg, w, other)[0][-1:], want[-1:]) > 10 * DTYPES["float32"]  # the first tokens do matter at the end
    m = load(ctx, tmp_path, dtype)
    for sizes in ([200], [2], [77, 1], [1]):
        assert off(portions(m, ids, sizes), want) <= DTYPES[dtype], sizes
    m.free()


def test_constants_are_read(ctx, tmp_path):
    """Every constant of the configuration changes the result the way it changes the oracle's."""
    base, w = build("ragged")
    ids = tokens(base, 60)
    ref, _ = D.forward(base, w, ids)
    changes = [lambda c: c["embedding"].update(scale=0.7), lambda c: c.update(logit_scale=3.0), lambda c: c["norm"].update(eps=0.3),
               lambda c: c["layers"][1]["mixer"]["mask"].update(size=7), lambda c: c["layers"][1]["mixer"]["rot"].update(base=3.0),
               lambda c: c["layers"][1]["mixer"].update(scale=0.05), lambda c: c["layers"][2]["mixer"]["mask"].update(size=51)]
    for i, change in enumerate(changes):
        cfg = json.loads(json.dumps(base))
        change(cfg)
        D.write_model(tmp_path / str(i), cfg, w)
        want, _ = D.forward(cfg, w, ids)
        assert np.abs(want - ref).max() > 1e-3
        m = load(ctx, tmp_path / str(i), "float32")
        got = m.feed(ids, 0, range(60))
        assert np.abs(got - want).max() <= 2e-4 * np.abs(want).max(), i
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


def follow(cfg, w, prompt, ids, tol):
    follows(D.forward, cfg, w, prompt, ids, tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["ragged", "tiles"])
def test_greedy_generation(ctx, folders, name, dtype):
    path, cfg, w = folders(name)
    tol = 4 * DTYPES[dtype]
    s = B.Session(ctx, path, B.Limits(ctx=400, max_tokens=32, kv=B.Dunuzen.kv_type(dtype)))
    prompt = tokens(cfg, 75, seed=3)
    ids, st = s.generate(prompt, 40)
    assert len(ids) == 40 and st.stop == "MaxTokens" and st.reused_tokens == 0
    follow(cfg, w, prompt, ids, tol)
    # the conversation goes on: all of it is reused; then a prompt that branches off: none of it
    more = np.concatenate([prompt, ids, tokens(cfg, 11, seed=8)])
    ids2, st2 = s.generate(more, 10)
    assert st2.reused_tokens == 115
    follow(cfg, w, more, ids2, tol)
    branch = np.concatenate([prompt[:50], tokens(cfg, 9, seed=2)])
    ids3, st3 = s.generate(branch, 10)
    assert st3.reused_tokens == 0
    follow(cfg, w, branch, ids3, tol)
    # device-resident loop through the model, and the callback and stop-id exits that leave a step queued ahead
    logits, _ = s.model.forward(prompt[:32], 0)
    s.model.forward(prompt[32:64], 32)
    logits, _ = s.model.forward(prompt[64:], 64)
    first = int(np.argmax(logits[0]))
    dev, _ = s.model.decode_greedy(first, 75, 12)
    assert [first] + list(dev[:11]) == list(ids[:12])
    s.reset()
    seen = []
    got, st = s.generate(prompt, 40, on_token=lambda t: (seen.append(t), len(seen) < 6)[1])
    assert st.stop == "Cancelled" and list(got) == list(ids[:6])
    cont = np.concatenate([prompt, ids[:6], tokens(cfg, 5, seed=1)])
    ids4, st4 = s.generate(cont, 8)
    assert st4.reused_tokens in (0, 80, 81)
    follow(cfg, w, cont, ids4, tol)
    s.free()


def test_sampled_generation(ctx, folders):
    """The device sampler behind this family draws what the host sampler draws from the same logits and stream."""
    path, cfg, w = folders("tiles")
    lim = B.Limits(ctx=200, max_tokens=64, kv=B.KvType.F32)
    params = B.SamplingParams(temperature=0.8, top_k=20, top_p=0.9, seed=5)
    s = B.Session(ctx, path, lim)
    prompt = tokens(cfg, 30)
    ids, _ = s.generate(prompt, 25, params)
    s.reset()
    again, _ = s.generate(prompt, 25, params)
    s.reset()
    s.set_stop_ids([cfg["vocab"] - 1], ignore_stop=True)  # masked: logits come to the host and its sampler draws
    host, _ = s.generate(prompt, 25, params)
    assert list(ids) == list(again)
    if cfg["vocab"] - 1 not in ids:
        assert sum(a == b for a, b in zip(ids, host)) >= 20
    s.free()


def test_graph_and_plain_steps_agree(ctx, folders):
    path, cfg, _ = folders("tiles")
    code = ("import sys, numpy as np; sys.path.insert(0, sys.argv[1]); import brasa_b200 as B; c = B.Context(0); "
            "m = B.Dunuzen.load_in(c, sys.argv[2], 'bfloat16', 200, 64); l, _ = m.forward(np.arange(50), 0); "
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
    want, _ = oracle(cfg, w, ids)
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
        assert off(got, want[rows]) <= DTYPES[dtype]
    assert not (tmp_path / "1.f32").exists()


def test_command_line_generates(ctx, folders):
    path, cfg, w = folders("tiles")
    prompt = tokens(cfg, 20)
    r = subprocess.run([sys.executable, "-m", "brasa_b200", "generate", str(path), "--prompt", ",".join(map(str, prompt)), "--max-new", "8", "--dtype", "float32"],
                       capture_output=True, text=True, cwd=ROOT, timeout=120)
    assert r.returncode == 0, r.stderr
    ids = np.array([int(t) for t in r.stdout.split()])
    assert len(ids) == 8
    follow(cfg, w, prompt, ids, 1e-3)


def test_qwen3_rows_of_logits(ctx, golden_dir):
    """forward_rows on the older family: any places of a run, the same numbers as the last rows."""
    m = B.Qwen3.load_in(ctx, golden_dir / "tiny" / "model.brasa", "float32", 64, 32, 8)
    ids = np.arange(3, 27)
    last, _ = m.forward(ids, 0, 4)
    assert np.array_equal(m.forward_rows(ids, 0, [20, 21, 22, 23]), last)
    mixed = m.forward_rows(ids, 0, [23, 2, 21])
    assert np.array_equal(mixed[[2, 0]], last[[1, 3]])
    m.free()
