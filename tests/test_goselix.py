"""Goselix without a GPU: configuration, weight layout, registry, and what the plain implementation
(oracle/goselix_ref.py) is sensitive to."""
import json

import numpy as np
import pytest

from caten_b200 import decoder, registry
from caten_b200 import goselix as M
from oracle import goselix_ref as R

import goselix_cases as K


# ---- configuration ----
def test_config_round_trip():
    c = M.parse_config(json.loads(json.dumps(K.CASES["mixed"])))
    assert (c.width, c.vocab, c.eps, c.loop) == (112, 151, 1e-5, (1, 3, 3))
    assert [type(l.mixer).__name__ for l in c.layers] == ["RetentionConfig", "LatentConfig", "LatentConfig", "RetentionConfig"]
    assert [type(l.mlp).__name__ for l in c.layers] == ["DenseConfig", "ExpertsConfig", "NoneType", "ExpertsConfig"]
    assert c.layers[1].mixer == M.LatentConfig(4, 24, 10, 16, 48, 80, 10000.0, 34 ** -0.5)
    assert c.layers[0].mixer == M.RetentionConfig(3, 20, 36, 12, 10000.0, (0.875, 0.9375, 0.96875))
    assert c.layers[0].mlp.ff == 56 and c.layers[1].mlp == M.ExpertsConfig(24, 4, 1)
    assert M.parse_config(K.CASES["latent"]).loop is None


def _with(layer, **change):
    cfg = json.loads(json.dumps(K.CASES["mixed"]))
    at = cfg["layers"][layer]
    for k, v in change.items():
        a, b = k.split("__")
        at[a][b] = v
    return cfg


@pytest.mark.parametrize("cfg", [
    {**K.CASES["mixed"], "architecture": "Other"},
    {**K.CASES["mixed"], "layers": [{"type": "conv", "mixer": {}, "mlp": None}]},
    {**K.CASES["mixed"], "loop": {"start": 3, "stop": 9, "times": 2}},
    {**K.CASES["mixed"], "loop": {"start": 1, "stop": 2, "times": 0}},
    _with(0, mlp__kind="sparse"), _with(0, mixer__decay=[0.5]), _with(1, mixer__rot={"base": 10.0, "dims": 4}), _with(1, mlp__router={"experts": 2, "top": 3}),
])
def test_config_refuses_what_it_does_not_know(cfg):
    with pytest.raises(ValueError):
        M.parse_config(cfg)


def test_registry():
    assert "Goselix" in registry.ARCHITECTURES


# ---- weight layout ----
def test_head_layouts():
    a = np.arange(3 * 30 * 7, dtype=np.uint16).reshape(90, 7) + 1
    p = M._head_parts(a, 3, (20, 10), 64)
    assert p.shape == (3 * 48, 64) and np.count_nonzero(p) == a.size
    assert (p.reshape(3, 48, 64)[:, :20, :7] == a.reshape(3, 30, 7)[:, :20]).all() and (p.reshape(3, 48, 64)[:, 32:42, :7] == a.reshape(3, 30, 7)[:, 20:]).all()
    t = M._head_transposed(a, 3, 30)
    assert t.shape == (3 * 16, 64) and np.count_nonzero(t) == a.size and (t.reshape(3, 16, 64)[:, :7, :30] == a.reshape(3, 30, 7).transpose(0, 2, 1)).all()


def test_frequencies():
    np.testing.assert_allclose(decoder.rope_frequencies(12, 300.0), [300.0 ** (-2.0 * i / 12) for i in range(6)], rtol=1e-14)


# ---- the plain implementation ----
def test_plain_rotation_pairs_the_halves_and_leaves_the_rest():
    x = np.arange(14.0).reshape(2, 7)
    y = R.rotate_halves(x, 4, 100.0, first_position=3)
    for t in range(2):
        for i in range(2):
            z = (x[t, i] + 1j * x[t, 2 + i]) * np.exp(1j * (3 + t) * 100.0 ** (-i / 2))
            np.testing.assert_allclose([y[t, i], y[t, 2 + i]], [z.real, z.imag], rtol=1e-12)
    assert (y[:, 4:] == x[:, 4:]).all()


def test_plain_recurrence_matches_its_unrolled_sum():
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((7, 4)), rng.standard_normal((7, 4)), rng.standard_normal((7, 5))
    o = R.retention_recurrence(q, k, v, 0.8)
    for t in range(7):
        np.testing.assert_allclose(o[t], sum(0.8 ** (t - s) * (q[t] @ k[s]) * v[s] for s in range(t + 1)), rtol=1e-10, atol=1e-12)


def test_plain_routing_and_input_weights():
    W = {"router": np.array([[1.0, 0.0], [0.0, 1.0], [1.0, 1.0]])}
    assert [e for e, _ in R.route(np.array([[2.0, 1.0]]), W, "", 2)[0]] == [2, 0]
    w = R.route(np.array([[2.0, 1.0]]), W, "", 1)[0][0][1]
    assert w == pytest.approx(1 / (1 + np.exp(-3.0)))
    rng = np.random.default_rng(1)
    W.update({f"e{e}.{n}": rng.standard_normal((2, 2)) for e in range(3) for n in ("gate", "up", "down")})
    h = np.array([[2.0, 1.0]])
    got = R.expert_mixture(h, W, "", {"router": {"top": 1}})
    np.testing.assert_allclose(got, R.silu_glu(w * h, W, "e2."), rtol=1e-12)
    assert np.abs(got - w * R.silu_glu(h, W, "e2.")).max() > 1e-3      # not the same as weighting the output


def test_plain_layer_runs():
    assert R.layer_runs(K.CASES["mixed"]) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert R.layer_runs(K.CASES["loop_all"]) == [(0, 0), (1, None), (0, 1), (1, None)]
    assert R.layer_runs(K.CASES["loop_once"]) == [(0, None), (1, 0)]


@pytest.mark.parametrize("kind", ["latent", "retention"])
def test_planted_pair_stands_out(kind):
    cfg = K.far_config(kind)
    t = K.plant(cfg, kind)
    toks = np.random.default_rng(2).integers(2, 40, 120)
    toks[-1] = 1
    a = R.forward(cfg, K.weights(t), toks)[-1]
    toks[5] = 0
    b = R.forward(cfg, K.weights(t), toks)[-1]
    toks[5], toks[70] = 3, 0
    c = R.forward(cfg, K.weights(t), toks)[-1]
    assert K.rel_rms(a[None], b[None])[0] > 0.3 and K.rel_rms(a[None], c[None])[0] > 0.3


@pytest.mark.parametrize("mistake", ["rotation", "shared_key", "latent_norm", "query_norm", "decay", "key_factor", "head_norm", "gate", "top", "output_weight", "loop", "step",
                                     "x0", "norm2", "sequential"])
def test_plain_implementation_shows_a_planted_mistake(mistake, monkeypatch):
    """Each mechanism moves the logits of the test model far beyond the tolerances of the GPU tests."""
    cfg, _, W = K.case("mixed")
    toks = K.tokens("mixed", 40)
    good = R.forward(cfg, W, toks)
    cfg, W = json.loads(json.dumps(cfg)), dict(W)
    if mistake == "rotation":
        monkeypatch.setattr(R, "rotate_halves", lambda x, dims, base, first_position=0: x)
    elif mistake == "shared_key":
        W["l1.mix.dkv"] = np.concatenate([W["l1.mix.dkv"][:80], np.zeros_like(W["l1.mix.dkv"][80:])])
    elif mistake in ("latent_norm", "query_norm"):
        orig, n = R.rms_norm, 80 if mistake == "latent_norm" else 48
        monkeypatch.setattr(R, "rms_norm", lambda x, g, eps: x * g if x.shape[-1] == n else orig(x, g, eps))
    elif mistake == "decay":
        for l in cfg["layers"]:
            if "decay" in l["mixer"]:
                l["mixer"]["decay"][0] -= 0.02
    elif mistake == "key_factor":
        # (a constant factor of k cancels in the heads' norm but for eps: small eps hides it, so it is made large)
        cfg["norm"]["eps"] = 1.0
        good = R.forward(cfg, W, toks)
        for l in cfg["layers"]:
            if "decay" in l["mixer"]:
                W.update({k: v * 2 for k, v in W.items() if k.endswith("mix.k")})
                break
    elif mistake == "head_norm":
        orig = R.rms_unit
        monkeypatch.setattr(R, "rms_unit", lambda x, eps: x if x.shape[-1] == 36 else orig(x, eps))
    elif mistake == "gate":
        orig = R.silu
        monkeypatch.setattr(R, "silu", lambda z: np.ones_like(z) if z.shape[-1] == 108 else orig(z))
    elif mistake == "top":
        cfg["layers"][1]["mlp"]["router"]["top"] = 2
    elif mistake == "output_weight":
        monkeypatch.setattr(R, "expert_mixture", lambda h, W, pre, spec: np.stack([sum(w * R.silu_glu(h[t:t + 1], W, f"{pre}e{e}.")[0] for e, w in ch)
                                                                                   for t, ch in enumerate(R.route(h, W, pre, spec["router"]["top"]))]))
    elif mistake == "loop":
        cfg["loop"]["times"] = 2
    elif mistake == "step":
        W["loop.step"] = np.roll(W["loop.step"], 1, axis=0)
    elif mistake == "x0":
        orig = R.layer_runs
        monkeypatch.setattr(R, "layer_runs", lambda c: [(i, t if t != 1 else 0) for i, t in orig(c)])
    elif mistake == "norm2":
        W["l0.norm2"] = W["l0.norm1"]
    elif mistake == "sequential":
        def layer(x, W, i, spec, eps):
            pre = f"l{i}."
            x = x + R.MIXERS[spec["type"]](R.rms_norm(x, W[pre + "norm1"], eps), W, pre + "mix.", spec["mixer"], eps)
            return x + R.feed_forward(R.rms_norm(x, W[pre + "norm2"], eps), W, pre + "mlp.", spec["mlp"]) if spec.get("mlp") else x
        monkeypatch.setattr(R, "layer", layer)
    assert K.rel_rms(R.forward(cfg, W, toks), good)[22:].max() > 5e-3
