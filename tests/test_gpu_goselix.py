"""Goselix and its mechanisms on the GPU against the plain implementation (oracle/goselix_ref.py)."""
import json
import os
import subprocess

import numpy as np
import pytest

import goselix_cases as K
from caten_b200 import _lib as L
from caten_b200 import goselix as M
from caten_b200 import safetensors
from caten_b200 import synthetic as S
from caten_b200.model import generate
from oracle import goselix_ref as R

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
LIMIT = {"fp32": 2e-5, "bf16x3": 3e-4, "bf16": 0.06}
NAMES = sorted(K.CASES)


def make(rt, name, precision="fp32", **kw):
    cfg, t, _ = K.case(name)
    return M.Goselix(rt, M.parse_config(cfg), t, precision=precision, **kw)


def feed(m, toks, cuts, first=0):
    """Logits of every token of ``toks``, in portions."""
    n, rows = first, []
    for c in cuts:
        rows.append(m.step(toks[n - first:n - first + c], n, range(c))[0][0])
        n += c
    assert n - first == len(toks)
    return np.concatenate(rows)


def check(got, want, precision, name=None, what=""):
    err = K.rel_rms(got, want)
    if precision == "bf16" and name and K.has_experts(name):
        # rounding decides between experts whose scores nearly tie: such a row, and a little of what follows, is another one
        assert np.quantile(err, 0.85) < LIMIT[precision] and np.median(err) < LIMIT[precision] / 2, (what, err.max())
    else:
        assert err.max() < LIMIT[precision], (what, err.max(), err.argmax())


# ---- whole models -------------------------------------------------------------------------------------
@pytest.mark.parametrize("precision", sorted(LIMIT))
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_portions_and_decoding(rt, name, precision):
    cfg, _, W = K.case(name)
    T = 150
    toks = K.tokens(name, T)
    want, layers = R.forward(cfg, W, toks, want_layers=True)
    m = make(rt, name, precision, max_seq_len=T, max_portion=150 if name != "mixed" else 48)
    check(feed(m, toks, [T]), want, precision, name)
    if name != "mixed" and not (precision == "bf16" and K.has_experts(name)):
        res = m.layer_outputs(toks)
        assert res.shape == layers.shape and np.abs(res - layers).max() < LIMIT[precision] * 10 * np.abs(layers).max()
    for cuts in ([2, 3, 2, 64, 1, 30, 48], [60] + [1] * 90, [1] * 7 + [143], [5] * 30, [2] * 75, [4, 4, 128, 4, 4, 4, 2]):
        check(feed(m, toks, cuts), want, precision, name, cuts)
    m.close()


def test_layers_after_each_token(rt):
    """The residual stream after every layer run, token by token, and the passes of a loop."""
    for name in ("mixed", "loop_all"):
        cfg, _, W = K.case(name)
        toks = K.tokens(name, 12, seed=8)
        _, layers = R.forward(cfg, W, toks, want_layers=True)
        m = make(rt, name, "fp32", max_seq_len=12)
        got = np.concatenate([m.layer_outputs(toks[i:i + 1], i) for i in range(12)], axis=1)
        assert got.shape == layers.shape and np.abs(got - layers).max() < 2e-5 * np.abs(layers).max()
        m.close()


def test_wanted_places_in_any_order(rt):
    cfg, _, W = K.case("mixed")
    toks = K.tokens("mixed", 100, seed=4)
    want = R.forward(cfg, W, toks)
    m = make(rt, "mixed", "fp32", max_seq_len=100, max_portion=32)
    got = m.step(toks, 0, [99, 0, 31, 32, 63, 5, 64])[0][0]
    assert K.rel_rms(got, want[[99, 0, 31, 32, 63, 5, 64]]).max() < LIMIT["fp32"]
    assert m.step(toks[:3], 0)[0].shape == (1, 0, cfg["vocab"])
    m.close()


@pytest.mark.parametrize("precision", sorted(LIMIT))
@pytest.mark.parametrize("name", ["dense", "mixed"])
def test_batch_equals_each_alone(rt, name, precision):
    cfg, _, W = K.case(name)
    B, T = 6, 60
    toks = np.stack([K.tokens(name, T, seed=s) for s in range(B)])
    m = make(rt, name, precision, max_seq_len=T, batch=B, max_rows=40, max_portion=13)   # several groups of sequences
    got = np.concatenate([m.step(toks[:, :41], 0, range(41))[0], m.step(toks[:, 41:43], 41, range(2))[0], m.step(toks[:, 43:58], 43, range(15))[0]] +
                         [m.step(toks[:, i:i + 1], i, [0])[0] for i in (58, 59)], axis=1)
    for b in range(B):
        check(got[b], R.forward(cfg, W, toks[b]), precision, name, b)
    m.close()


def test_sequences_follow_one_another(rt):
    """A new sequence sees nothing of the ones before it, whatever their lengths."""
    for precision in ("fp32", "bf16x3"):
        m = make(rt, "mixed", precision, max_seq_len=200)
        cfg, _, W = K.case("mixed")
        for i, (T, first) in enumerate([(120, 100), (1, 1), (30, 1), (90, 2), (2, 2), (64, 64)]):
            toks = K.tokens("mixed", T, seed=10 + i)
            check(feed(m, toks, [first] + [1] * (T - first)), R.forward(cfg, W, toks), precision)
        m.close()


def test_long_decoding(rt):
    for name, T in (("mixed", 300), ("dense", 420)):
        cfg, _, W = K.case(name)
        toks = K.tokens(name, T, seed=3)
        want = R.forward(cfg, W, toks)
        for precision in ("fp32", "bf16"):
            m = make(rt, name, precision, max_seq_len=T, max_portion=16)
            check(feed(m, toks, [16] + [1] * (T - 16)), want, precision, name)
            m.close()


def test_cache_sizes(rt):
    """Latent layers hold kv_rank + rot_dim numbers a token, retention layers a state, whatever the heads are."""
    m = make(rt, "latent", "bf16", max_seq_len=100)
    assert m.cache_nbytes == 128 * (48 + 16) * 2
    assert make(rt, "dense", "bf16", max_seq_len=129, batch=3).cache_nbytes == 3 * (256 * (64 + 32) * 2 + 2 * 32 * 64 * 4)   # rot_dim 16 stored as 32
    m.close()
    m = make(rt, "latent", "fp32", max_seq_len=100)
    assert m.cache_nbytes == 128 * (48 + 16) * 4
    m.close()
    a, b = (make(rt, "retention", "bf16", max_seq_len=t) for t in (10, 5000))
    assert a.cache_nbytes == b.cache_nbytes == 4 * 32 * 48 * 4
    a.close(); b.close()


# ---- latent attention and retention: a pair that stands out --------------------------------------------
@pytest.mark.parametrize("precision", sorted(LIMIT))
@pytest.mark.parametrize("kind", ["latent", "retention"])
def test_far_token_is_found(rt, kind, precision):
    """Token 1 asks for token 0, once in each sequence, on both sides of the borders of the kernels' tiles and chunks; asked for
    in a prompt, at the start of a portion, in a portion of two and in decoding."""
    cfg = K.far_config(kind)
    t = K.plant(cfg, kind)
    W, T = K.weights(t), 420
    m = M.Goselix(rt, M.parse_config(cfg), t, precision=precision, max_seq_len=T)
    rng = np.random.default_rng(5)
    for at in (0, 1, 31, 32, 63, 64, 65, 127, 128, 129, 255, 256, 300):
        toks = rng.integers(2, 40, T)
        toks[at] = 0
        asked = [q for q in (at + 1, 64, 128, 129, 256, 257, 383, 384, 400, 401, 418, 419) if q > at]
        toks[asked] = 1
        want = R.forward(cfg, W, toks)
        for cuts in ([T], [128, 128, 128, 36], [400] + [1] * 20, [382, 2, 2, 2, 12, 2, 18]):
            check(feed(m, toks, cuts)[asked], want[asked], precision, None, (at, cuts))
    m.close()


@pytest.mark.parametrize("capacity", [420, 9000])
def test_latent_decoding_with_key_splits(rt, capacity):
    """Few sequences split the keys over CTAs, some of which may have none; the result must not depend on it."""
    cfg = K.far_config("latent")
    t = K.plant(cfg, "latent")
    W, T = K.weights(t), 420
    toks = np.random.default_rng(6).integers(2, 40, T)
    toks[3] = 0
    toks[[4, 100, 128, 300, 400, 410, 419]] = 1
    want = R.forward(cfg, W, toks)
    for precision in sorted(LIMIT):
        m = M.Goselix(rt, M.parse_config(cfg), t, precision=precision, max_seq_len=capacity)
        check(feed(m, toks, [3] + [1] * 130 + [2] * 40 + [1] * (T - 213)), want, precision)
        m.close()


def test_retention_decays_from_forgetting_to_remembering(rt):
    """Decays of exactly 1 and close to 0 side by side, over more than one chunk."""
    cfg = S.goselix_config(64, 50, "r-", 16, 1, 16, 16, 16, 16, 16, 4, 32, 64, 16, decay=(1.0, 0.999999, 1e-3, 1e-30))
    t = S.synth_goselix(cfg, seed=9)
    toks = np.random.default_rng(1).integers(0, 50, 300)
    want = R.forward(cfg, K.weights(t), toks)
    m = M.Goselix(rt, M.parse_config(cfg), t, precision="fp32", max_seq_len=300)
    for cuts in ([300], [65, 63, 64, 2, 106], [128] + [1] * 172):
        check(feed(m, toks, cuts), want, "fp32", None, cuts)
    m.close()


@pytest.mark.parametrize("H,D,P,E,K_", [(1, 16, 16, 16, 16), (16, 48, 16, 64, 128), (17, 32, 32, 32, 64), (33, 16, 2, 16, 200), (128, 16, 16, 16, 320), (3, 40, 24, 56, 500)])
def test_latent_shapes(rt, H, D, P, E, K_):
    """Head counts on both sides of a CTA's, latents of one block to many."""
    cfg = S.goselix_config(64, 30, "l-", 16, H, D, P, E, 32, K_, 1, 16, 16, 16)
    t = S.synth_goselix(cfg, seed=H + K_)
    B, T = 3, 140
    toks = np.random.default_rng(H).integers(0, 30, (B, T))
    want = [R.forward(cfg, K.weights(t), toks[b]) for b in range(B)]
    for precision in ("bf16", "bf16x3"):
        m = M.Goselix(rt, M.parse_config(cfg), t, precision=precision, max_seq_len=T, batch=B)
        got = np.concatenate([m.step(toks[:, :126], 0, range(126))[0], m.step(toks[:, 126:130], 126, range(4))[0]] + [m.step(toks[:, i:i + 1], i, [0])[0] for i in range(130, T)], axis=1)
        for b in range(B):
            check(got[b], want[b], precision)
        m.close()


@pytest.mark.parametrize("H,D,E,rot", [(1, 16, 16, 16), (8, 64, 128, 64), (3, 128, 256, 100), (2, 200, 64, 2), (1, 48, 520, 48)])
def test_retention_shapes(rt, H, D, E, rot):
    cfg = S.goselix_config(64, 30, "r-", 16, 1, 16, 16, 16, 16, 16, H, D, E, rot)
    t = S.synth_goselix(cfg, seed=H + D)
    B, T = 2, 150
    toks = np.random.default_rng(D).integers(0, 30, (B, T))
    m = M.Goselix(rt, M.parse_config(cfg), t, precision="fp32", max_seq_len=T, batch=B)
    got = np.concatenate([m.step(toks[:, :129], 0, range(129))[0], m.step(toks[:, 129:131], 129, range(2))[0]] + [m.step(toks[:, i:i + 1], i, [0])[0] for i in range(131, T)], axis=1)
    for b in range(B):
        check(got[b], R.forward(cfg, K.weights(t), toks[b]), "fp32")
    m.close()


# ---- experts ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("experts,top,ff", [(1, 1, 16), (3, 3, 40), (8, 2, 130), (33, 5, 16), (300, 3, 8)])
@pytest.mark.parametrize("precision", ["fp32", "bf16x3"])
def test_expert_mixtures(rt, experts, top, ff, precision):
    """From one token (one row per pair) to many rows per expert, experts without rows, every expert of a token."""
    cfg = S.goselix_config(64, 60, "rm", 16, 1, 16, 16, 16, 16, 16, 1, 16, 16, 16, experts=experts, top=top, expert_ff=ff)
    t = S.synth_goselix(cfg, seed=experts)
    T = 700
    toks = np.random.default_rng(top).integers(0, 60, T)
    want = R.forward(cfg, K.weights(t), toks)
    m = M.Goselix(rt, M.parse_config(cfg), t, precision=precision, max_seq_len=T)
    for cuts in ([T], [1, 2, 3, 4, 5, 6, 16, 33, 64, 130, 300, 136]):
        check(feed(m, toks, cuts), want, precision, None, cuts)
    m.close()


# ---- batches --------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name,B", [("mixed", 5), ("mixed", 40), ("mixed", 300), ("loop_once", 5), ("loop_once", 40)])
def test_decoding_batches(rt, name, B):
    """Row tiles, key splits, expert tiles and the form of the per-head products change with the batch; a sequence's result does not."""
    cfg, _, W = K.case(name)
    T = 24
    toks = np.stack([K.tokens(name, T, seed=s) for s in range(B)])
    want = [R.forward(cfg, W, toks[b]) for b in range(0, B, max(1, B // 4))]
    for precision in ("fp32", "bf16x3"):
        m = make(rt, name, precision, max_seq_len=T, batch=B)
        got = np.concatenate([m.step(toks[:, :9], 0, range(9))[0]] + [m.step(toks[:, i:i + 1], i, [0])[0] for i in range(9, 20)] + [m.step(toks[:, 20:], 20, range(4))[0]], axis=1)
        for i, b in enumerate(range(0, B, max(1, B // 4))):
            check(got[b], want[i], precision, None, b)
        m.close()


def test_many_rows_of_many_heads(rt):
    """More than a thousand sequences: the per-head products run on the many-row linear, whose tiles do not line up with heads."""
    cfg = S.goselix_config(64, 30, "l-", 16, 40, 16, 16, 16, 32, 48, 1, 16, 16, 16)
    t = S.synth_goselix(cfg, seed=1)
    B, T = 1100, 6
    toks = np.random.default_rng(0).integers(0, 30, (B, T))
    want = {b: R.forward(cfg, K.weights(t), toks[b]) for b in (0, 1, 500, 1023, 1024, 1099)}
    for precision in ("bf16", "bf16x3"):
        m = M.Goselix(rt, M.parse_config(cfg), t, precision=precision, max_seq_len=T, batch=B)
        got = np.concatenate([m.step(toks[:, :2], 0, range(2))[0]] + [m.step(toks[:, i:i + 1], i, [0])[0] for i in range(2, T)], axis=1)
        for b, w in want.items():
            check(got[b], w, precision, None, b)
        m.close()


# ---- generation, errors, commands -----------------------------------------------------------------------
@pytest.mark.parametrize("name", ["mixed", "loop_once", "experts"])
def test_greedy_generation(rt, name):
    cfg, _, W = K.case(name)
    prompt = K.tokens(name, 9, seed=1)
    m = make(rt, name, "fp32", max_seq_len=40)
    got = generate(m, prompt, 25)[0]
    lg = R.forward(cfg, W, got)
    top2 = np.sort(lg, axis=1)[:, -2:]
    decisive = top2[8:-1, 1] - top2[8:-1, 0] > 1e-3 * np.abs(lg).max()
    assert decisive.sum() > 15 and (got[9:] == lg[8:-1].argmax(axis=1))[decisive].all()
    first = m.forward(prompt, 9, 0)
    assert (m.decode_device(first, 9, 24)[0] == got[10:]).all()     # ids stay on the device
    sampled = generate(m, prompt, 10, temperature=0.8, top_k=5, seed=2)
    assert (sampled == generate(m, prompt, 10, temperature=0.8, top_k=5, seed=2)).all() and (sampled < cfg["vocab"]).all()
    m.close()
    mb = make(rt, name, "fp32", max_seq_len=40, batch=5)
    batch = np.stack([K.tokens(name, 9, seed=1 + i) for i in range(5)])
    out = generate(mb, batch, 25)
    assert (out[0] == got).mean() > 0.9 and (out[0][:12] == got[:12]).all()
    mb.close()


def test_step_errors(rt):
    m = make(rt, "dense", "fp32", max_seq_len=16)
    m.step([1, 2, 3], 0)
    for bad in (lambda: m.step([1], 2), lambda: m.step([1], 4), lambda: m.step([1] * 14, 3), lambda: m.step([1], -1), lambda: m.step([1, 2], 3, [2])):
        with pytest.raises(L.B200Error):
            bad()
    assert m.step([4], 3, [0])[0].shape == (1, 1, 203)     # still where it was
    m.close()


def test_missing_and_misshapen_tensors_are_refused(rt):
    cfg, t, _ = K.case("experts")
    for name, change in (("l0.mix.dkv", None), ("l1.mlp.e4.down", None), ("head", np.zeros((90, 129), np.uint16)), ("l0.norm2", np.zeros(2, np.uint16)),
                         ("l0.mlp.router", np.zeros((4, 128), np.uint16))):
        bad = dict(t)
        if change is None:
            del bad[name]
        else:
            bad[name] = change
        with pytest.raises((KeyError, ValueError)):
            M.Goselix(rt, M.parse_config(cfg), bad, max_seq_len=8)


@pytest.fixture(scope="module")
def stored(tmp_path_factory):
    cfg, t, W = K.case("mixed")
    d = tmp_path_factory.mktemp("model")
    (d / "config.json").write_text(json.dumps(cfg))
    safetensors.save(str(d / "model.safetensors"), t)
    return str(d), cfg, W


@pytest.mark.parametrize("dtype,precision", [("float32", "fp32"), ("bfloat16", "bf16")])
def test_trace_run(stored, tmp_path, dtype, precision):
    path, cfg, W = stored
    a, b = K.tokens("mixed", 70, seed=5), K.tokens("mixed", 33, seed=6)
    steps, expect, wa, wb = [], {}, R.forward(cfg, W, a), R.forward(cfg, W, b)
    for rid, toks, ref, cuts in (("x", a, wa, [0, 40, 42, 43, 70]), ("y", b, wb, [0, 1, 33])):
        for lo, hi in zip(cuts, cuts[1:]):
            want = list(range(hi - lo))
            expect[len(steps)] = ref[lo:hi]
            steps.append({"step": len(steps), "entries": [{"id": rid, "tokens": toks[lo:hi].tolist(), "want": want}], "end": [rid] if hi == len(toks) else []})
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "80"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600, cwd=ROOT)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    got = np.concatenate([np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(ref.shape) for i, ref in expect.items()])
    check(got, np.concatenate(list(expect.values())), precision, "mixed")


def test_generate_command(stored, capsys):
    from caten_b200.generate import main
    path, cfg, W = stored
    assert main(["--model", path, "--ids", "5,17,3", "--max-length", "6", "--precision", "fp32"]) == 0
    ids = [int(x) for x in capsys.readouterr().out.strip().split(",")]
    assert ids[:3] == [5, 17, 3] and ids == R.greedy(cfg, W, [5, 17, 3], 6)
