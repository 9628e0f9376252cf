"""Gugedra without a GPU: the float64 oracle against scalar loops, the registry, refusals and the memory plan."""

import json
import math

import numpy as np
import pytest

import brasa_b200 as B
from brasa_b200 import __main__ as cli
from oracle import dunuzen as D
from oracle import gugedra as G

from dunuzen_cases import tokens
from gugedra_cases import CASES, attn, build, config, delta, parallel, ssm


# ---- the oracle, each mechanism against plain loops ----------------------------------------------------------------------


def test_gelu_and_softcap():
    for z in (-3.0, -0.2, 0.0, 1.7):
        assert np.isclose(G.gelu_tanh(np.array(z)), 0.5 * z * (1 + math.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3))))
    assert np.isclose(G.softcap(np.array(50.0), 30.0), 30 * math.tanh(50 / 30)) and abs(G.softcap(np.array(1e-3), 30.0) - 1e-3) < 1e-9


def test_grouped_rms_norms_every_part_alone():
    x = np.array([[3.0, 4.0, 100.0, 0.0]])
    y = G.grouped_rms(x, 2, 0.0)
    assert np.allclose(y, [[3 / math.sqrt(12.5), 4 / math.sqrt(12.5), math.sqrt(2), 0.0]])
    assert np.allclose(G.grouped_rms(x, 1, 0.0), x / math.sqrt((9 + 16 + 1e4) / 4))


def test_state_space_scan_scalar():
    rng = np.random.default_rng(3)
    x, Bm, C = rng.standard_normal((5, 1)), rng.standard_normal((5, 2)), rng.standard_normal((5, 2))
    dt, a_log, d = rng.uniform(0.1, 2, 5), -0.4, 0.7
    out, S = G.state_space_scan(x, Bm, C, dt, a_log, d, np.zeros((2, 1)))
    s = [0.0, 0.0]
    for t in range(5):
        f = math.exp(-math.exp(a_log) * dt[t])
        s = [f * s[n] + dt[t] * Bm[t, n] * x[t, 0] for n in range(2)]
        assert np.isclose(out[t, 0], s[0] * C[t, 0] + s[1] * C[t, 1] + d * x[t, 0])
    assert np.allclose(S[:, 0], s)


def test_attention_heads_share_keys_and_windows_end():
    cfg = attn(4, 2, 6, 3, 3, 4, softcap=5.0)
    rng = np.random.default_rng(1)
    w = {n: rng.standard_normal(s) for n, s in (("q", (24, 5)), ("k", (12, 5)), ("v", (6, 5)), ("o", (5, 12)))}
    h = rng.standard_normal((7, 5))
    got = G.window_attention(h, w.__getitem__, cfg)

    def rotated(v, p):
        v = list(v)
        for i in range(2):
            a = p * 1000.0 ** (-2 * i / 4)
            v[i], v[i + 2] = v[i] * math.cos(a) - v[i + 2] * math.sin(a), v[i + 2] * math.cos(a) + v[i] * math.sin(a)
        return np.array(v)
    for t in range(7):
        cat = []
        for head in range(4):
            g = head // 2
            q = rotated((w["q"] @ h[t])[6 * head:6 * head + 6], t)
            seen = [j for j in range(7) if 0 <= t - j < 3]
            s = [5.0 * math.tanh(q @ rotated((w["k"] @ h[j])[6 * g:6 * g + 6], j) * cfg["scale"] / 5.0) for j in seen]
            p = np.exp(s) / np.sum(np.exp(s))
            cat.append(sum(p[i] * (w["v"] @ h[j])[3 * g:3 * g + 3] for i, j in enumerate(seen)))
        assert np.allclose(got[t], w["o"] @ np.concatenate(cat))


@pytest.mark.parametrize("name", list(CASES))
def test_oracle_is_causal(name):
    cfg, w = build(name)
    ids = tokens(cfg, 40)
    whole, _ = G.forward(cfg, w, ids)
    part, _ = G.forward(cfg, w, ids[:25])
    assert np.allclose(whole[:25], part, atol=1e-9) and np.abs(whole).max() < cfg["logit_softcap"]


# ---- folder, registry, plan ----------------------------------------------------------------------------------------------


@pytest.fixture()
def folder(tmp_path):
    cfg, w = build("ragged")
    D.write_model(tmp_path / "m", cfg, w)
    return tmp_path / "m", cfg, w


def test_registry_chooses_the_class(folder):
    path, cfg, w = folder
    assert B.model_class(path) is B.Gugedra
    shape, c = B.model_shape(path)
    assert (c["hidden"], c["layers"], c["vocab"]) == (cfg["width"], len(cfg["layers"]), cfg["vocab"])
    assert shape.weight_bytes >= sum(2 * v.size for v in w.values())


@pytest.mark.parametrize("change, message", [
    (lambda c: c.pop("logit_softcap"), "logit_softcap"),
    (lambda c: c.update(logit_softcap=0.0), "positive"),
    (lambda c: c["token_side"].update(dim=6), "unexpected"),
    (lambda c: c["layers"][0].update(type="parallel"), "left is missing"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "feed-forward"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("softcap"), "softcap"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(norm_groups=7), "norm_groups"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(groups=4), "multiple of groups"),
    (lambda c: c["layers"][1]["mixer"].pop("right_scale"), "right_scale"),
    (lambda c: c["layers"][0].update(mlp=None) or c["layers"][3].update(mlp={"kind": "dense", "ff": 9}), "missing tensor"),
])
def test_bad_configurations_are_refused(folder, change, message):
    path, cfg, _ = folder
    cfg = json.loads(json.dumps(cfg))
    change(cfg)
    (path / "config.json").write_text(json.dumps(cfg))
    with pytest.raises(B.BrasaError) as e:
        B.model_shape(path)
    assert message in str(e.value)


def test_plan_follows_the_window_not_the_context(tmp_path):
    cfg = config(64, 50, [(parallel(attn(4, 2, 16, 8, 40, 16), ssm(4, 8, 16, 1, 1, 4)), 64), (delta(2, 2, 16, 16, 4), None)])
    D.write_model(tmp_path, cfg, G.random_weights(cfg, 0))

    def plan(ctx, kv=B.KvType.BF16):
        return B.planner.check_path(None, tmp_path, B.Limits(ctx=ctx, max_tokens=100, kv=kv), 1 << 40)[1]
    short, long, f32 = plan(16), plan(100000), plan(100000, B.KvType.F32)
    assert short["kv"] < long["kv"] == plan(200000)["kv"]   # the ring is bounded by window + run
    rows = 256                                              # 40 - 1 + 100 rounded up to 128
    assert long["kv"] < f32["kv"] <= long["kv"] + rows * 2 * (16 + 8) * 2 + 4096


def test_cli_info(folder, capsys):
    assert cli.main(["info", str(folder[0])]) == 0
    assert "family Gugedra" in capsys.readouterr().out
