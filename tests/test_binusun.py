"""Binusun without a GPU: configuration, frequencies, weight layout, file reader, registry, trace replay,
and what the plain implementation (oracle/binusun_ref.py) is sensitive to."""
import io
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from caten_b200 import binusun as M
from caten_b200 import registry, safetensors, trace
from caten_b200.safetensors import SafeTensors, bf16_to_f32, f32_to_bf16
from oracle import binusun_ref as R

import binusun_cases as K

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ---- configuration ----
def test_config_round_trip():
    cfg = K.CASES["mixed"][0]
    c = M.parse_config(json.loads(json.dumps(cfg)))
    assert (c.width, c.vocab, c.eps, c.logit_scale, c.loop) == (160, 203, 1e-5, 1.5, (1, 3, 2))
    assert [type(l.mixer).__name__ for l in c.layers] == ["WkvConfig", "AttentionConfig", "AttentionConfig", "WkvConfig"]
    assert [l.ff for l in c.layers] == [None, 96, None, 96]
    a = c.layers[1].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.rot_dims, a.rot_base, a.scale) == (6, 2, 40, 24, 21, 12, 500.0, 40 ** -0.5)
    assert a.rot_scaling == (8.0, 1.0, 4.0, 256.0)
    assert M.parse_config(K.CASES["attention"][0]).loop is None and M.parse_config(K.CASES["attention"][0]).layers[0].mixer.rot_scaling is None


@pytest.mark.parametrize("change", [
    {"architecture": "Other"},
    {"layers": [{"type": "conv", "mixer": {}, "mlp": None}]},
    {"layers": [{"type": "wkv", "mixer": {"heads": 1, "dim": 16}, "mlp": {"kind": "sparse", "ff": 4}}]},
    {"loop": {"start": 3, "stop": 9, "times": 2}},
    {"loop": {"start": 1, "stop": 2, "times": 0}},
])
def test_config_refuses_what_it_does_not_know(change):
    with pytest.raises(ValueError):
        M.parse_config({**K.CASES["mixed"][0], **change})


@pytest.mark.parametrize("dims,base,scaling", [(2, 10000.0, None), (24, 10000.0, K.SCALING), (64, 500000.0, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}),
                                               (20, 1000.0, {"factor": 2.0, "low": 0.5, "high": 8.0, "original": 64}), (16, 10000.0, {"factor": 1.0, "low": 1.0, "high": 4.0, "original": 100})])
def test_rope_frequencies(dims, base, scaling):
    got = M.rope_frequencies(dims, base, [scaling[k] for k in ("factor", "low", "high", "original")] if scaling else None)
    want = R.rope_frequencies(dims, base, scaling)
    np.testing.assert_allclose(got, want, rtol=1e-14)
    if scaling and scaling["factor"] != 1.0:   # all three branches occur
        plain = R.rope_frequencies(dims, base)
        wl, o = 2 * np.pi / plain, scaling["original"]
        assert (wl < o / scaling["high"]).any() and (wl > o / scaling["low"]).any()


# ---- weight layout ----
def test_head_layouts():
    a = np.arange(3 * 20 * 7, dtype=np.uint16).reshape(60, 7) + 1
    r = M._head_rows(a, 3, 20, 64)
    assert r.shape == (96, 64) and (r.reshape(3, 32, 64)[:, :20, :7] == a.reshape(3, 20, 7)).all() and np.count_nonzero(r) == a.size
    c = M._head_cols(np.ascontiguousarray(a.T), 3, 20, 64)
    assert c.shape == (64, 128) and (c[:7, :96].reshape(7, 3, 32)[:, :, :20] == a.T.reshape(7, 3, 20)).all() and np.count_nonzero(c) == a.size
    v = M._head_vec(np.arange(60, dtype=np.float32) + 1, 3, 20)
    assert v.shape == (128,) and (v[:96].reshape(3, 32)[:, :20].reshape(-1) == np.arange(60) + 1).all() and np.count_nonzero(v) == 60


# ---- files ----
def test_safetensors_round_trip(tmp_path):
    p = str(tmp_path / "t.safetensors")
    t = {"a": np.arange(6, dtype=np.uint16).reshape(2, 3), "b": np.float32([[1.5]]), "s": f32_to_bf16(np.float32(-2.0)), "i": np.int32([7, 8])}
    safetensors.save(p, t)
    st = SafeTensors(p)
    assert sorted(st.names()) == ["a", "b", "i", "s"] and "a" in st and "x" not in st
    assert (st.bf16("a") == t["a"]).all() and st.f32("b") == 1.5 and st.bf16("s").shape == () and float(st.f32("s")) == -2.0
    assert (st.raw("i") == t["i"]).all() and st.dtype("i") == "I32"
    with pytest.raises(ValueError):
        st.bf16("b")
    with pytest.raises(KeyError):
        st.raw("x")


def test_safetensors_refuses_damaged_files(tmp_path):
    p = str(tmp_path / "t.safetensors")
    safetensors.save(p, {"a": np.zeros((4, 4), np.float32)})
    b = open(p, "rb").read()
    for bad in (b[:4], b[:-8], b"\xff" * 8 + b[8:]):
        open(p, "wb").write(bad)
        with pytest.raises(ValueError):
            SafeTensors(p)


def test_bf16_rounds_to_nearest_even():
    x = np.float32([1.0, 1.0 + 2 ** -8, 1.0 + 3 * 2 ** -8, 1.0 + 2 ** -8 + 2 ** -20, -3.14159])
    assert bf16_to_f32(f32_to_bf16(x)).tolist() == [1.0, 1.0, 1.015625, 1.0078125, -3.140625]


def test_registry(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Nothing"}))
    assert registry.architecture_of(str(tmp_path)) == "Nothing"
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.load_model(str(tmp_path), runtime=object())
    assert {"gpt2", "Binusun"} <= set(registry.ARCHITECTURES)


# ---- trace replay ----
class FakeModel:
    def __init__(self):
        self.calls = []

    def step(self, tok, n, want=()):
        self.calls.append((tok[0].tolist(), n, list(want)))
        return np.float32([[[10 * n + w, tok[0][w]] for w in want]]), None


def test_replay_feeds_portions_in_order():
    m = FakeModel()
    r = trace.Replay(m)
    assert r.step([{"id": "a", "tokens": [5, 6, 7], "want": []}], []) is None
    assert r.step([{"id": "a", "tokens": [8, 9], "want": [1, 0]}], ["a"]).tolist() == [[31, 9], [30, 8]]
    assert r.step([{"id": "b", "tokens": [1], "want": [0]}], []).tolist() == [[0, 1]]
    assert m.calls == [([5, 6, 7], 0, []), ([8, 9], 3, [1, 0]), ([1], 0, [0])]
    with pytest.raises(ValueError):
        r.step([{"id": "c", "tokens": [1], "want": [0]}], [])


def test_replay_main_writes_files(tmp_path, monkeypatch, capsys):
    class Rt:
        def __enter__(self): return self
        def __exit__(self, *a): pass
    fake = FakeModel()
    fake.close = lambda: None
    monkeypatch.setattr(trace, "B200Runtime", lambda d: Rt())
    monkeypatch.setattr(trace, "load_model", lambda *a, **k: fake)
    monkeypatch.setattr(sys, "stdin", io.StringIO('{"step": 3, "entries": [{"id": "a", "tokens": [4, 5], "want": [1]}], "end": ["a"]}\n\n{"step": 4, "entries": [], "end": []}\n'))
    assert trace.main(["--model", "m", "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "8"]) == 0
    assert capsys.readouterr().out == "done 3\ndone 4\n"
    assert np.fromfile(tmp_path / "3.f32", "<f4").tolist() == [1.0, 5.0] and os.listdir(tmp_path) == ["3.f32"]


def test_commands_show_help():
    for cmd in ([os.path.join(ROOT, "bin", "trace_run"), "--help"], [sys.executable, "-m", "caten_b200.generate", "--help"]):
        r = subprocess.run(cmd, cwd=ROOT, capture_output=True, text=True, timeout=300)
        assert r.returncode == 0 and "--model" in r.stdout, r.stderr


# ---- the plain implementation ----
def test_plain_rotation_is_interleaved_and_leaves_the_rest():
    x = np.arange(12.0).reshape(2, 6)
    y = R.rotate(x, np.array([0.5, 0.25]), first_position=3)
    for t in range(2):
        for i, f in enumerate((0.5, 0.25)):
            z = (x[t, 2 * i] + 1j * x[t, 2 * i + 1]) * np.exp(1j * (3 + t) * f)
            np.testing.assert_allclose(y[t, 2 * i:2 * i + 2], [z.real, z.imag], rtol=1e-12)
    assert (y[:, 4:] == x[:, 4:]).all()


def test_plain_window_edges():
    q, k, v = np.zeros((6, 2)), np.zeros((6, 2)), np.eye(6)
    q[:, 0], k[1, 0] = 1.0, 50.0                     # key 1 stands out
    o = R.window_attention(q, k, v, 3, 1.0)
    assert np.allclose(o[1:4, 1], 1.0) and np.allclose(o[4], [0, 0, 1 / 3, 1 / 3, 1 / 3, 0]) and np.allclose(o[0, 0], 1.0)
    # a window one token off shows at exactly one query
    off = R.window_attention(q, k, v, 4, 1.0)
    assert np.flatnonzero(np.abs(off - o).max(axis=1) > 0.5).tolist() == [4]


def test_plain_recurrence_matches_its_unrolled_sum():
    rng = np.random.default_rng(0)
    r, k, v = rng.standard_normal((3, 7, 4))
    w, u = rng.uniform(0.1, 1.0, (7, 4)), rng.standard_normal(4)
    o = R.wkv_recurrence(r, k, v, w, u)
    for t in range(7):
        want = (r[t] * u * k[t]).sum() * v[t]
        for s in range(t):
            want = want + (r[t] * np.prod(w[s + 1:t], axis=0) * k[s]).sum() * v[s]
        np.testing.assert_allclose(o[t], want, rtol=1e-10, atol=1e-12)


def test_plain_layer_runs():
    assert R.layer_runs(K.CASES["mixed"][0]) == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert R.layer_runs(K.CASES["loop_once"][0]) == [(0, False), (1, False), (2, True)]
    assert R.layer_runs(K.CASES["wkv"][0]) == [(0, False)]


@pytest.mark.parametrize("mistake", ["window", "rotation", "qk_norm", "gate", "bonus", "decay", "shift", "loop", "scaling", "post_norm"])
def test_plain_implementation_shows_a_planted_mistake(mistake, monkeypatch):
    """Each mechanism moves the logits of the test model far beyond the tolerances of the GPU tests."""
    cfg, _, W = K.case("mixed")
    toks = K.tokens("mixed", 40)
    good = R.forward(cfg, W, toks)
    cfg, W = json.loads(json.dumps(cfg)), dict(W)
    if mistake == "window":
        for l in cfg["layers"]:
            if "mask" in l["mixer"]:
                l["mixer"]["mask"]["size"] += 1
    elif mistake == "rotation":
        monkeypatch.setattr(R, "rotate", lambda x, f, first_position=0: x)
    elif mistake == "qk_norm":
        orig = R.rms_unit
        monkeypatch.setattr(R, "rms_unit", lambda x, eps: x if x.shape[-1] == 40 else orig(x, eps))
    elif mistake == "gate":
        W.update({k: np.zeros_like(v) for k, v in W.items() if k.endswith("mix.g") and v.shape[0] == 6})
    elif mistake == "bonus":
        W.update({k: np.zeros_like(v) for k, v in W.items() if k.endswith("mix.u")})
    elif mistake == "decay":
        W.update({k: np.zeros_like(v) for k, v in W.items() if k.endswith("mix.w2")})
    elif mistake == "shift":
        monkeypatch.setattr(R, "token_shift", lambda h, mu: h)
    elif mistake == "loop":
        cfg["loop"]["times"] = 1
    elif mistake == "scaling":
        for l in cfg["layers"]:
            if "rot" in l["mixer"]:
                l["mixer"]["rot"]["scaling"] = None
    elif mistake == "post_norm":
        W["l1.norm1b"] = W["l1.norm1b"] * 1.1
    assert K.rel_rms(R.forward(cfg, W, toks), good)[22:].max() > 5e-3
