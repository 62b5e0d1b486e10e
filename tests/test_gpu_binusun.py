"""Binusun and its mechanisms on the GPU against the plain implementation (oracle/binusun_ref.py)."""
import json
import os
import subprocess

import numpy as np
import pytest

import binusun_cases as K
from caten_b200 import _lib as L
from caten_b200 import binusun as M
from caten_b200 import safetensors
from caten_b200.model import generate
from caten_b200.safetensors import bf16_to_f32, f32_to_bf16
from caten_b200.synthetic import Packed
from oracle import binusun_ref as R

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def p16(n):
    return -(-n // 16) * 16


def make(rt, name, precision="fp32", **kw):
    cfg, t, _ = K.case(name)
    return M.Binusun(rt, M.parse_config(cfg), t, precision=precision, **kw)


def bf16_weight(rt, rng, rows, cols):
    bits = f32_to_bf16(rng.standard_normal((rows, cols), dtype=np.float32) * np.float32(cols ** -0.5))
    return rt.upload_weight(Packed(L.BF16, rows, cols, bits.view(np.uint8).reshape(-1))), bf16_to_f32(bits).astype(np.float64)


# ---- linears over bf16 weights, plain and gated -----------------------------------------------------
SHAPES = [(1, 77, 64), (3, 130, 320), (7, 77, 128), (40, 256, 1024), (300, 130, 192), (1100, 4868, 64), (1024, 2432, 128)]


@pytest.mark.parametrize("M_,N,Kd", SHAPES)
@pytest.mark.parametrize("precision", ["fp32", "bf16", "bf16x3"])
def test_linear_bf16_weight(rt, M_, N, Kd, precision):
    rng = np.random.default_rng(M_ + N)
    w, wf = bf16_weight(rt, rng, N, Kd)
    x = rng.standard_normal((M_, Kd), dtype=np.float32)
    assert (w.dequantize() == wf.astype(np.float32)).all() and w.device_nbytes == 2 * N * Kd
    got = rt.linear(w, rt.transfer_from_array(x), precision=L.PRECISIONS[precision]).numpy()
    assert np.abs(got - x @ wf.T).max() < (3e-2 if precision == "bf16" else 1e-4)


@pytest.mark.parametrize("M_,N,Kd", [(m, n + n % 2, k) for m, n, k in SHAPES])
@pytest.mark.parametrize("precision", ["fp32", "bf16", "bf16x3"])
def test_gated_linear(rt, M_, N, Kd, precision):
    rng = np.random.default_rng(M_ + N + 1)
    w, wf = bf16_weight(rt, rng, N, Kd)
    x, bias = rng.standard_normal((M_, Kd), dtype=np.float32), rng.standard_normal(N, dtype=np.float32)
    y = x @ wf.T + bias
    want = np.maximum(y[:, 0::2], 0) * y[:, 1::2]
    got = rt.linear(w, rt.transfer_from_array(x), bias=rt.transfer_from_array(bias), act=L.ACT_RELU_GLU, precision=L.PRECISIONS[precision],
                    out=rt.open_buffer((M_, N // 2))).numpy()
    assert np.abs(got - want).max() < (0.15 if precision == "bf16" else 4e-4)


def test_gated_linear_refuses_what_it_cannot_do(rt):
    rng = np.random.default_rng(0)
    w, _ = bf16_weight(rt, rng, 77, 64)
    with pytest.raises(L.B200Error):
        rt.linear(w, rt.open_buffer((2, 64)), act=L.ACT_RELU_GLU, out=rt.open_buffer((2, 38)))


# ---- windowed grouped-query attention ----------------------------------------------------------------
class AttnCase:
    """Random projections of `s` tokens for B sequences, the ring caches, and the plain result."""

    def __init__(self, rt, H, G, D, E, window, s, B=1, rot=None, qk_norm=1, gated=1, scale=0.3, cap=None, seed=0, tweak=None):
        rng = np.random.default_rng(seed + H + 7 * D + 13 * window)
        self.rt, self.B, self.s, self.H, self.G, self.D, self.E = rt, B, s, H, G, D, E
        rot = D // 2 * 2 if rot is None else rot
        freqs = R.rope_frequencies(rot, 1000.0)
        q, k = rng.standard_normal((B, s, H, D)), rng.standard_normal((B, s, G, D))
        v, g = rng.standard_normal((B, s, G, E)), rng.standard_normal((B, s, H))
        if tweak:
            tweak(q, k, v)
        q, k, v, g = (np.asarray(a, np.float32) for a in (q, k, v, g))
        Dp, Ep = p16(D), p16(E)
        self.ld = -(-(H * Dp + G * (Dp + Ep) + (H if gated else 0)) // 64) * 64
        qkv = np.zeros((B, s, self.ld), np.float32)
        qkv[..., :H * Dp].reshape(B, s, H, Dp)[..., :D] = q
        qkv[..., H * Dp:(H + G) * Dp].reshape(B, s, G, Dp)[..., :D] = k
        o = (H + G) * Dp
        qkv[..., o:o + G * Ep].reshape(B, s, G, Ep)[..., :E] = v
        if gated:
            qkv[..., o + G * Ep:o + G * Ep + H] = g
        self.qkv = qkv
        eps = 1e-5
        self.want = np.zeros((B, s, H, E))
        for b in range(B):
            for h in range(H):
                kv = h // (H // G)
                qa, ka = R.rotate(q[b, :, h].astype(np.float64), freqs), R.rotate(k[b, :, kv].astype(np.float64), freqs)
                if qk_norm:
                    qa, ka = R.rms_unit(qa, eps), R.rms_unit(ka, eps)
                self.want[b, :, h] = R.window_attention(qa, ka, v[b, :, kv].astype(np.float64), window or s, scale)
                if gated:
                    self.want[b, :, h] *= R.sigmoid(g[b, :, h:h + 1].astype(np.float64))
        self.freq = rt.transfer_from_array(freqs.astype(np.float32)) if rot else None
        self.desc = L.AttnDesc(H, G, D, E, window, rot, qk_norm, gated, scale, eps, self.freq.ptr if rot else None)
        self.cap = cap or -(-s // 64) * 64
        self.kc, self.vc = rt.open_buffer((B, G, self.cap, Dp)), rt.open_buffer((B, G, self.cap, Ep))

    def run(self, portions, precision):
        got, n = np.zeros_like(self.want), 0
        for c in portions:
            x = self.rt.transfer_from_array(np.ascontiguousarray(self.qkv[:, n:n + c]).reshape(self.B * c, self.ld))
            o = self.rt.attn_window(self.desc, x, self.kc, self.vc, self.B, c, n, L.PRECISIONS[precision]).numpy()
            got[:, n:n + c] = o.reshape(self.B, c, self.H, -1)[..., :self.E]
            n += c
        assert n == self.s
        return got


ATTN = [  # H, G, D, E, window
    (2, 2, 64, 64, 5), (4, 2, 64, 64, 64), (4, 1, 32, 64, 65), (3, 3, 40, 24, 33), (4, 2, 96, 128, 70), (2, 1, 128, 40, 127), (8, 2, 16, 16, 1),
    (2, 1, 64, 64, 0), (4, 1, 136, 200, 50), (6, 1, 80, 112, 300)]


@pytest.mark.parametrize("H,G,D,E,window", ATTN)
@pytest.mark.parametrize("precision", ["fp32", "bf16x3"])
def test_attention_prompts_portions_and_decoding(rt, H, G, D, E, window, precision):
    s = 210
    c = AttnCase(rt, H, G, D, E, window, s, rot=D // 4 * 2)
    for portions in ([s], [2, 63, 1, 64, 65, 3, 12], [130] + [1] * 80, [1] * 20 + [190]):
        np.testing.assert_allclose(c.run(portions, precision), c.want, atol=4e-5, rtol=0, err_msg=str(portions))


@pytest.mark.parametrize("precision", ["fp32", "bf16x3"])
@pytest.mark.parametrize("window,portion", [(20, 45), (64, 64), (100, 29)])
def test_attention_ring_is_reused_many_times(rt, window, portion, precision):
    s = 900
    c = AttnCase(rt, 2, 1, 48, 64, window, s, B=2, cap=-(-(window - 1 + portion) // 64) * 64)
    sizes, left, i = [], s, 0
    while left:
        k = min(left, [portion, 1, 7, portion, 1, 1, 2][i % 7])
        sizes.append(k)
        left -= k
        i += 1
    # angles are fp32: at position 900 their rounding (900 * 2^-24) alone moves q and k by 5e-5
    np.testing.assert_allclose(c.run(sizes, precision), c.want, atol=1.5e-4, rtol=0)
    with pytest.raises(L.B200Error):   # a portion the ring cannot hold beside the window
        rt.attn_window(c.desc, rt.open_buffer((2 * (c.cap + 1), c.ld)), c.kc, c.vc, 2, c.cap + 1, s, L.PREC_FP32)


@pytest.mark.parametrize("window", [3, 64, 65, 100, 128])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("precision", ["fp32", "bf16x3"])
def test_attention_window_edge_stands_out(rt, window, decode, precision):
    """One key outweighs all others for every query: it is the answer as long as it is inside the window and
    absent one token later, in prompts and in decoding, wherever it lies relative to blocks of keys."""
    s = window + 150
    for j0 in (0, 1, 63, 64, 100):
        def tweak(q, k, v):
            q[...] = 0.0
            k[...] = 0.0
            v[...] = 0.0
            q[..., 0] = 1.0
            k[:, j0, :, 0] = 40.0
            v[:, j0, :, :] = 1.0
        c = AttnCase(rt, 2, 1, 64, 64, window, s, rot=0, qk_norm=0, gated=0, scale=1.0, tweak=tweak)
        got = c.run([j0 + 1] + [1] * (s - j0 - 1) if decode else [s], precision)[0, :, :, 0]
        inside = slice(j0, j0 + window)
        assert np.abs(got[inside] - 1.0).max() < 1e-4, (j0, window)
        assert np.abs(got[j0 + window:]).max() < 1e-4 and (j0 == 0 or np.abs(got[:j0]).max() < 1e-4)


@pytest.mark.parametrize("precision", ["fp32", "bf16x3"])
def test_attention_far_key_among_hundreds(rt, precision):
    s = 700
    def tweak(q, k, v):
        k[:, 17] = 0.0
        k[:, 17, :, 40:] = 6.0          # beyond the rotated dims
        q[:, 600:, :, 40:] = 6.0        # aligned with key 17 only
        v[:, 17] = 3.0
    c = AttnCase(rt, 4, 2, 64, 48, 650, s, rot=40, qk_norm=0, gated=0, scale=0.02, tweak=tweak)
    assert (c.want[0, 600:660] > 2.9).all() and (c.want[0, 680:] < 2.0).all()
    for portions in ([s], [600] + [1] * 100, [333, 2, 365]):
        np.testing.assert_allclose(c.run(portions, precision), c.want, atol=1e-4, rtol=0)


def test_attention_batch_equals_each_alone(rt):
    for precision in ("fp32", "bf16x3"):
        c = AttnCase(rt, 8, 2, 64, 64, 37, 120, B=5, cap=128)
        got = c.run([50, 2, 60] + [1] * 8, precision)
        np.testing.assert_allclose(got, c.want, atol=4e-5, rtol=0)


@pytest.mark.parametrize("B,G,rep", [(1, 1, 1), (1, 2, 4), (70, 2, 4), (200, 1, 8), (90, 2, 2)])
def test_attention_decode_launch_shapes(rt, B, G, rep):
    """Head groups per CTA and key splits over a cluster change with the batch; the result must not."""
    c = AttnCase(rt, G * rep, G, 32, 48, 90, 96, B=B, cap=128)
    np.testing.assert_allclose(c.run([93, 1, 1, 1], "bf16x3"), c.want, atol=4e-5, rtol=0)


# ---- time mixing --------------------------------------------------------------------------------------
class WkvCase:
    def __init__(self, rt, H, D, s, B=1, low=64, seed=0, w0=-2.0, spread=1.5):
        rng = np.random.default_rng(seed + H + D)
        self.rt, self.B, self.s, self.H, self.D, Dp = rt, B, s, H, D, p16(D)
        self.Dp = Dp
        gr = -(-H * Dp // 128) * 128
        hd = -(-H * Dp // 64) * 64
        r, k, v, g = (rng.standard_normal((B, s, H, D)).astype(np.float32) for _ in range(4))
        x = rng.standard_normal((B, s, low)).astype(np.float32)
        w2 = f32_to_bf16(rng.standard_normal((H, D, low)).astype(np.float32) * np.float32(low ** -0.5))
        w0 = (w0 + spread * rng.standard_normal((H, D))).astype(np.float32)
        u, norm = (rng.standard_normal((H, D)).astype(np.float32) for _ in range(2))
        y = np.zeros((B, s, 4 * gr + low), np.float32)
        for i, a in enumerate((r, k, v, g)):
            y[..., i * gr:i * gr + H * Dp].reshape(B, s, H, Dp)[..., :D] = a
        y[..., 4 * gr:] = x
        self.y = y
        d = np.tanh(x.astype(np.float64)) @ bf16_to_f32(w2).astype(np.float64).reshape(H * D, low).T
        decay = np.exp(-np.exp(d.reshape(B, s, H, D) + w0))
        self.want = np.zeros((B, s, H, D))
        for b in range(B):
            for h in range(H):
                o = R.wkv_recurrence(*(a[b, :, h].astype(np.float64) for a in (r, k, v)), decay[b, :, h], u[h].astype(np.float64))
                self.want[b, :, h] = R.rms_unit(o, 1e-5) * norm[h] * R.silu(g[b, :, h].astype(np.float64))
        pad = np.zeros((H, Dp, low), np.uint16)
        pad[:, :D] = w2
        pad = np.concatenate([pad.reshape(H * Dp, low), np.zeros((hd - H * Dp, low), np.uint16)])
        self.w2 = rt.upload_weight(Packed(L.BF16, hd, low, pad.view(np.uint8).reshape(-1)))
        def vec(a):
            out = np.zeros((H, Dp), np.float32)
            out[:, :D] = a
            return rt.transfer_from_array(out)
        self.vecs = [vec(a) for a in (w0, u, norm)]
        self.desc = L.WkvDesc(H, D, gr, low, 1e-5, *(a.ptr for a in self.vecs), self.w2.handle)
        self.state = rt.transfer_from_array(np.full((B, H, Dp, Dp), 7.0, np.float32))   # a new sequence must not read it

    def run(self, portions, precision="fp32"):
        got, n = np.zeros_like(self.want), 0
        for c in portions:
            y = self.rt.transfer_from_array(np.ascontiguousarray(self.y[:, n:n + c]).reshape(self.B * c, -1))
            o = self.rt.wkv(self.desc, y, self.state, self.B, c, n, L.PRECISIONS[precision]).numpy()
            got[:, n:n + c] = o[:, :self.H * self.Dp].reshape(self.B, c, self.H, self.Dp)[..., :self.D]
            n += c
        assert n == self.s
        return got


@pytest.mark.parametrize("H,D,B", [(2, 64, 1), (3, 16, 2), (1, 40, 1), (2, 100, 1), (1, 128, 2), (1, 200, 1), (1, 256, 1), (40, 64, 8), (16, 32, 40)])
def test_time_mixing_prompts_portions_and_decoding(rt, H, D, B):
    s = 150
    c = WkvCase(rt, H, D, s, B=B)
    for portions in ([s], [2, 15, 16, 17, 1, 64, 33, 2], [100] + [1] * 50, [1] * 10 + [140]):
        got = c.run(portions)
        # a head's output can be small before its norm: compare on the scale of the head
        np.testing.assert_allclose(got, c.want, atol=3e-4, rtol=2e-3, err_msg=str(portions))


@pytest.mark.parametrize("w0,spread", [(-9.0, 0.5), (3.0, 1.0), (-2.0, 6.0)])
def test_time_mixing_extreme_decays(rt, w0, spread):
    """Memories of thousands of tokens, of less than one token, and both side by side."""
    c = WkvCase(rt, 2, 64, 300, w0=w0, spread=spread)
    for portions in ([300], [129, 2, 100, 69]):
        np.testing.assert_allclose(c.run(portions), c.want, atol=5e-4, rtol=4e-3)


def test_time_mixing_long_memory(rt):
    """A token far back is still in the state: its value comes out when its key is asked for again."""
    c = WkvCase(rt, 1, 64, 400, w0=-12.0, spread=0.0)
    y = c.y.reshape(400, -1)
    gr = c.desc.group_rows
    y[:, gr:gr + 64] *= 0.01
    y[5, gr:gr + 64] = 2.0
    c.y = y.reshape(1, 400, -1)
    r, k, v, g = (y[:, i * gr:i * gr + 64].astype(np.float64) for i in range(4))
    w2 = c.w2.dequantize()[:64].astype(np.float64)
    w = np.exp(-np.exp(np.tanh(y[:, 4 * gr:].astype(np.float64)) @ w2.T + c.vecs[0].numpy()[0]))
    o = R.wkv_recurrence(r, k, v, w, c.vecs[1].numpy()[0].astype(np.float64))
    want = R.rms_unit(o, 1e-5) * c.vecs[2].numpy()[0] * R.silu(g)
    for portions in ([400], [200] + [1] * 200):
        np.testing.assert_allclose(c.run(portions)[0, :, 0], want, atol=5e-4, rtol=4e-3)


# ---- whole models -------------------------------------------------------------------------------------
LIMIT = {"fp32": 2e-5, "bf16x3": 3e-4, "bf16": 0.06}
NAMES = sorted(K.CASES)


@pytest.mark.parametrize("precision", sorted(LIMIT))
@pytest.mark.parametrize("name", NAMES)
def test_model_whole_prompts_portions_and_decoding(rt, name, precision):
    cfg, _, W = K.case(name)
    T = 150
    toks = K.tokens(name, T)
    want, layers = R.forward(cfg, W, toks, want_layers=True)
    m = make(rt, name, precision, max_seq_len=T, max_portion=150 if name != "mixed" else 48)
    every = list(range(T))
    got = m.step(toks, 0, every)[0][0]
    assert K.rel_rms(got, want).max() < LIMIT[precision]
    if name != "mixed":
        res = m.layer_outputs(toks)
        assert res.shape == layers.shape and np.abs(res - layers).max() < LIMIT[precision] * 10 * np.abs(layers).max()
    for portions in ([2, 3, 2, 64, 1, 30, 48], [60] + [1] * 90, [1] * 7 + [143], [5] * 30):
        n, rows = 0, []
        for c in portions:
            rows.append(m.step(toks[n:n + c], n, range(c))[0][0])
            n += c
        assert n == T and K.rel_rms(np.concatenate(rows), want).max() < LIMIT[precision], portions
    m.close()


def test_model_wanted_places_in_any_order(rt):
    cfg, _, W = K.case("mixed")
    toks = K.tokens("mixed", 100, seed=4)
    want = R.forward(cfg, W, toks)
    m = make(rt, "mixed", "fp32", max_seq_len=100, max_portion=32)
    got = m.step(toks, 0, [99, 0, 31, 32, 63, 5, 64])[0][0]
    assert K.rel_rms(got, want[[99, 0, 31, 32, 63, 5, 64]]).max() < LIMIT["fp32"]
    assert m.step(toks[:3], 0)[0].shape == (1, 0, cfg["vocab"])
    m.close()


@pytest.mark.parametrize("precision", ["fp32", "bf16"])
def test_model_batch_equals_each_alone(rt, precision):
    cfg, _, W = K.case("loop_all")
    B, T = 6, 60
    toks = np.stack([K.tokens("loop_all", T, seed=s) for s in range(B)])
    m = make(rt, "loop_all", precision, max_seq_len=T, batch=B, max_rows=40, max_portion=13)   # several groups of sequences
    got = np.concatenate([m.step(toks[:, :41], 0, range(41))[0], m.step(toks[:, 41:58], 41, range(17))[0]] +
                         [m.step(toks[:, i:i + 1], i, [0])[0] for i in (58, 59)], axis=1)
    for b in range(B):
        assert K.rel_rms(got[b], R.forward(cfg, W, toks[b])).max() < LIMIT[precision]
    m.close()


def test_model_sequences_follow_one_another(rt):
    """A new sequence sees nothing of the ones before it, whatever their lengths."""
    m = make(rt, "mixed", "fp32", max_seq_len=200)
    cfg, _, W = K.case("mixed")
    for i, (T, first) in enumerate([(120, 100), (1, 1), (30, 1), (90, 2), (2, 2), (64, 64)]):
        toks = K.tokens("mixed", T, seed=10 + i)
        rows = [m.step(toks[:first], 0, range(first))[0][0]] + [m.step(toks[n:n + 1], n, [0])[0][0] for n in range(first, T)]
        assert K.rel_rms(np.concatenate(rows), R.forward(cfg, W, toks)).max() < LIMIT["fp32"]
    m.close()


def test_model_long_decoding(rt):
    cfg, _, W = K.case("mixed")
    T = 420
    toks = K.tokens("mixed", T, seed=3)
    want = R.forward(cfg, W, toks)
    for precision in ("fp32", "bf16"):
        m = make(rt, "mixed", precision, max_seq_len=T, max_portion=16)
        rows = [m.step(toks[:16], 0, range(16))[0][0]] + [m.step(toks[n:n + 1], n, [0])[0][0] for n in range(16, T)]
        assert K.rel_rms(np.concatenate(rows), want).max() < LIMIT[precision]
        m.close()


def test_windowed_caches_do_not_grow_with_the_sequence(rt):
    a, b = (make(rt, "attention", "fp32", max_seq_len=t, max_portion=64) for t in (1000, 100000))
    assert a.cache_nbytes == b.cache_nbytes == 2 * 128 * (32 + 32) * 4   # two key/value heads, a ring of p64(9 - 1 + 64)
    a.close(); b.close()


@pytest.mark.parametrize("name", ["mixed", "loop_once", "wkv"])
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
    m = make(rt, "wkv", "fp32", max_seq_len=16)
    m.step([1, 2, 3], 0)
    for bad in (lambda: m.step([1], 2), lambda: m.step([1], 4), lambda: m.step([1] * 14, 3), lambda: m.step([1], -1), lambda: m.step([1, 2], 3, [2])):
        with pytest.raises(L.B200Error):
            bad()
    assert m.step([4], 3, [0])[0].shape == (1, 1, 100)     # still where it was
    m.close()


def test_missing_and_misshapen_tensors_are_refused(rt):
    cfg, t, _ = K.case("wkv")
    for name, change in (("l0.mix.u", None), ("head", np.zeros((100, 65), np.uint16)), ("l0.norm1", np.zeros(2, np.uint16))):
        bad = dict(t)
        if change is None:
            del bad[name]
        else:
            bad[name] = change
        with pytest.raises((KeyError, ValueError)):
            M.Binusun(rt, M.parse_config(cfg), bad, max_seq_len=8)


# ---- the commands -------------------------------------------------------------------------------------
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
            want = [hi - lo - 1] + ([0] if hi - lo > 2 else [])
            if lo == 40:
                want = []
            else:
                expect[len(steps)] = ref[[lo + w for w in want]]
            steps.append({"step": len(steps), "entries": [{"id": rid, "tokens": toks[lo:hi].tolist(), "want": want}], "end": [rid] if hi == len(toks) else []})
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "80"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600, cwd=ROOT)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    assert sorted(os.listdir(tmp_path)) == sorted(f"{i}.f32" for i in expect)
    for i, ref in expect.items():
        got = np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(ref.shape)
        assert K.rel_rms(got, ref).max() < LIMIT[precision]


def test_generate_command(stored, capsys):
    from caten_b200.generate import main
    path, cfg, W = stored
    assert main(["--model", path, "--ids", "5,17,3", "--max-length", "6", "--precision", "fp32"]) == 0
    ids = [int(x) for x in capsys.readouterr().out.strip().split(",")]
    assert ids[:3] == [5, 17, 3] and ids == R.greedy(cfg, W, [5, 17, 3], 6)
