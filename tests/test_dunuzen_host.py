"""Dunuzen without a GPU: the float64 oracle against scalar loops, the model folder reader, the registry, the memory plan, the
trace runner's protocol and the command line."""

import io
import json
import math

import numpy as np
import pytest

import brasa_b200 as B
from brasa_b200 import __main__ as cli
from brasa_b200 import trace
from oracle import dunuzen as D

from dunuzen_cases import CASES, CD, LA, build, config, delta, latent, tokens


# ---- the oracle, each mechanism against plain loops ----------------------------------------------------------------------


def test_rope_pairs_and_positions():
    x = np.random.default_rng(0).standard_normal((3, 2, 10))
    y = D.rope_half(x, [0, 5, 9], 6, 50.0)
    assert np.allclose(y[0], x[0]) and np.array_equal(y[..., 6:], x[..., 6:])
    for t, p in enumerate([0, 5, 9]):
        for i in range(3):
            a = p * 50.0 ** (-2 * i / 6)
            assert np.allclose(y[t, :, i], x[t, :, i] * math.cos(a) - x[t, :, i + 3] * math.sin(a))
            assert np.allclose(y[t, :, i + 3], x[t, :, i + 3] * math.cos(a) + x[t, :, i] * math.sin(a))


def test_causal_conv_looks_back_taps_minus_one():
    x, w = np.zeros((6, 1)), np.array([[0.5, 2.0, 3.0]])
    x[1] = 1.0
    assert np.array_equal(D.causal_conv(x, w)[:, 0], [0, 3.0, 2.0, 0.5, 0, 0])


def test_delta_scan_scalar():
    rng = np.random.default_rng(3)
    q, k, v = rng.standard_normal((4, 2)), rng.standard_normal((4, 2)), rng.standard_normal((4, 1))
    g, beta = rng.uniform(0.2, 1, (4, 2)), rng.uniform(0, 1, 4)
    out, S = D.delta_scan(q, k, v, g, beta, np.zeros((2, 1)))
    a = b = 0.0
    for t in range(4):
        a, b = a * g[t, 0], b * g[t, 1]
        u = beta[t] * (v[t, 0] - a * k[t, 0] - b * k[t, 1])
        a, b = a + k[t, 0] * u, b + k[t, 1] * u
        assert np.isclose(out[t, 0], a * q[t, 0] + b * q[t, 1])
    assert np.allclose(S[:, 0], [a, b])


def test_delta_rule_overwrites_a_key():
    """With beta 1, no decay and a unit key, reading the key returns the last value written to it."""
    k = np.array([[0.6, 0.8], [0.6, 0.8]])
    out, _ = D.delta_scan(k, k, np.array([[3.0], [-7.0]]), np.ones((2, 2)), np.ones(2), np.zeros((2, 1)))
    assert np.allclose(out[:, 0], [3.0, -7.0])


@pytest.mark.parametrize("name", list(CASES))
def test_oracle_is_causal_and_windows_end(name):
    cfg, w = build(name)
    ids = tokens(cfg, 40)
    whole, _ = D.forward(cfg, w, ids)
    part, _ = D.forward(cfg, w, ids[:25])
    assert np.allclose(whole[:25], part, atol=1e-9)


def test_window_edge_in_oracle():
    seen = D.window_visible(9, 4)
    assert seen[8, 5] and not seen[8, 4] and seen[3, 0] and not seen[4, 0] and not seen[2, 3] and seen[0, 0]


# ---- folder, registry, plan ----------------------------------------------------------------------------------------------


@pytest.fixture()
def folder(tmp_path):
    cfg, w = build("ragged")
    D.write_model(tmp_path / "m", cfg, w)
    return tmp_path / "m", cfg, w


def test_registry_chooses_the_class(folder, golden_dir):
    path, cfg, w = folder
    assert B.model_class(path) is B.Dunuzen
    assert B.model_class(golden_dir / "tiny" / "model.brasa") is B.Qwen3
    shape, c = B.model_shape(path)
    assert (c["hidden"], c["layers"], c["vocab"]) == (cfg["width"], len(cfg["layers"]), cfg["vocab"])
    assert shape.weight_bytes >= sum(2 * v.size for v in w.values())


def rewrite(path, cfg, change):
    cfg = json.loads(json.dumps(cfg))
    change(cfg)
    (path / "config.json").write_text(json.dumps(cfg))


@pytest.mark.parametrize("change, message", [
    (lambda c: c.update(architecture="Nothing"), "not supported"),
    (lambda c: c.pop("width"), "width"),
    (lambda c: c.update(width=c["width"] + 8), "unexpected"),
    (lambda c: c["layers"][0].update(type="other"), "unknown mixer"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "feed-forward"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"].append(c["layers"][0]), "missing tensor"),
])
def test_bad_configurations_are_refused(folder, change, message):
    path, cfg, _ = folder
    rewrite(path, cfg, change)
    with pytest.raises(B.BrasaError) as e:
        B.model_shape(path)
        B.model_class(path)
    assert message in str(e.value)


def test_damaged_files_are_refused(folder):
    path, _, _ = folder
    data = (path / "model.safetensors").read_bytes()
    for cut in (4, 40, len(data) - 2):
        (path / "model.safetensors").write_bytes(data[:cut])
        with pytest.raises(B.BrasaError):
            B.model_shape(path)
    (path / "config.json").write_text("{")
    with pytest.raises(B.BrasaError):
        B.model_class(path)


def test_plan_follows_the_window_not_the_context(tmp_path):
    cfg = config(64, 50, [(LA, latent(2, 16, 8, 16, 32, 40), 64), (CD, delta(2, 2, 16, 16, 4), 64)])
    D.write_model(tmp_path, cfg, D.random_weights(cfg, 0))

    def plan(ctx, kv=B.KvType.BF16, budget=1 << 40):
        return B.planner.check_path(None, tmp_path, B.Limits(ctx=ctx, max_tokens=32, kv=kv), budget)
    short, long, f32 = plan(16)[1], plan(100000)[1], plan(100000, B.KvType.F32)[1]
    assert short["kv"] < long["kv"] == plan(200000)[1]["kv"]      # the ring is bounded by window + run
    rows = 128                                                    # 40 - 1 + 32 rounded up to 64
    assert long["kv"] < f32["kv"] <= long["kv"] + rows * (32 + 8) * 2 + 4096
    ok, p, largest = plan(1 << 20, budget=long["total"])
    assert not ok and 0 < largest < 1 << 20
    with pytest.raises(B.BrasaError):
        plan(64, B.KvType.F16)


def test_brasa_file_plans_through_the_same_call(golden_dir):
    path = golden_dir / "tiny" / "model.brasa"
    lim = B.Limits(ctx=64, max_tokens=16)
    shape, _ = B.model_shape(path)
    assert B.planner.check_path(None, path, lim, 1 << 40)[1] == B.planner.plan(shape, lim)


# ---- trace runner and command line ---------------------------------------------------------------------------------------


class FakeModel(B.Model):
    """Logits of a token: (token, its position)."""

    def __init__(self, max_tokens, max_rows):
        self.limits, self.cfg, self.runs = B.Limits(ctx=999, max_tokens=max_tokens, max_logit_rows=max_rows), {"head_rows": 2}, []

    def forward_rows(self, ids, pos0, rows):
        assert len(ids) <= self.limits.max_tokens and len(rows) <= self.limits.max_logit_rows
        self.runs.append((pos0, len(ids)))
        return np.array([[ids[r], pos0 + r] for r in rows], np.float32).reshape(len(rows), 2)


def replay(steps, tmp_path, model):
    said = []
    trace.replay(model, io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"), tmp_path, said.append)
    return said


def test_trace_protocol(tmp_path):
    m = FakeModel(4, 2)
    said = replay([{"step": 0, "entries": [{"id": "a", "tokens": [9, 8, 7, 6, 5, 4], "want": [5, 0, 1]}], "end": []},
                   {"step": 1, "entries": [{"id": "a", "tokens": [3], "want": []}], "end": ["a"]},
                   {"step": 2, "entries": [{"id": "b", "tokens": [1, 2], "want": [1]}], "end": ["b"]}], tmp_path, m)
    assert said == ["done 0", "done 1", "done 2"]
    assert np.array_equal(np.fromfile(tmp_path / "0.f32", "<f4").reshape(-1, 2), [[4, 5], [9, 0], [8, 1]])
    assert not (tmp_path / "1.f32").exists()
    assert np.array_equal(np.fromfile(tmp_path / "2.f32", "<f4"), [2, 1])
    assert m.runs == [(0, 4), (4, 2), (6, 1), (0, 2)]


def test_trace_refuses_interleaved_requests(tmp_path):
    with pytest.raises(ValueError):
        replay([{"step": 0, "entries": [{"id": "a", "tokens": [1], "want": []}], "end": []},
                {"step": 1, "entries": [{"id": "b", "tokens": [1], "want": []}], "end": []}], tmp_path, FakeModel(4, 2))


def test_feed_cuts_at_tokens_and_rows():
    m = FakeModel(8, 2)
    got = m.feed(np.arange(100, 120), 30, [0, 1, 2, 3, 19])
    assert np.array_equal(got, [[100, 30], [101, 31], [102, 32], [103, 33], [119, 49]])
    assert sum(n for _, n in m.runs) == 20 and all(b[0] == a[0] + a[1] for a, b in zip(m.runs, m.runs[1:]))


def test_cli_info(folder, capsys):
    assert cli.main(["info", str(folder[0])]) == 0
    assert "family Dunuzen" in capsys.readouterr().out
