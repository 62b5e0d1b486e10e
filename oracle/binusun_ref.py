"""Plain statement of the Binusun decoder in numpy: whole sequences, no cache, no state carried
between calls, loops over tokens and heads.  Test infrastructure; shares no code with the package.

``cfg`` is the parsed config.json of a model, ``W`` maps tensor names to arrays.  Every function
works in the dtype of its inputs (float64 unless a caller passes something else).
"""
from __future__ import annotations

import math

import numpy as np


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def scalar_norm(x, g, eps):
    """RMS norm whose gain is one number for all coordinates."""
    return rms_unit(x, eps) * np.asarray(g, x.dtype).reshape(())


def rope_frequencies(dims, base, scaling=None):
    """Angle per position of each interleaved pair; ``scaling`` as in Llama 3.1 (None: unscaled)."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            wavelength = 2.0 * math.pi / f
            factor, lo, hi, orig = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
            if wavelength < orig / hi:
                pass
            elif wavelength > orig / lo:
                f = f / factor
            else:
                s = (orig / wavelength - lo) / (hi - lo)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return np.array(out, np.float64)


def rotate(x, freqs, first_position=0):
    """x [tokens, dim]: the first 2 * len(freqs) dims are rotated as interleaved pairs."""
    y = x.copy()
    for t in range(x.shape[0]):
        for i, f in enumerate(freqs):
            a = (first_position + t) * f
            c, s = math.cos(a), math.sin(a)
            u, v = x[t, 2 * i], x[t, 2 * i + 1]
            y[t, 2 * i] = u * c - v * s
            y[t, 2 * i + 1] = v * c + u * s
    return y


def window_attention(q, k, v, window, scale):
    """One head: query i sees keys j with 0 <= i - j < window; ordinary softmax."""
    out = np.zeros((q.shape[0], v.shape[1]), q.dtype)
    for i in range(q.shape[0]):
        j0 = max(0, i - window + 1)
        s = (k[j0:i + 1] @ q[i]) * scale
        p = np.exp(s - s.max())
        out[i] = (p / p.sum()) @ v[j0:i + 1]
    return out


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def attention_mixer(h, W, pre, mx, eps):
    H, G, D, E = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q, k, v, gate = h @ W[pre + "q"].T, h @ W[pre + "k"].T, h @ W[pre + "v"].T, sigmoid(h @ W[pre + "g"].T)
    freqs = rope_frequencies(mx["rot"]["dims"], mx["rot"]["base"], mx["rot"].get("scaling"))
    heads = []
    for a in range(H):
        g = a // (H // G)
        qa = rms_unit(rotate(q[:, a * D:(a + 1) * D], freqs), eps)
        ka = rms_unit(rotate(k[:, g * D:(g + 1) * D], freqs), eps)
        o = window_attention(qa, ka, v[:, g * E:(g + 1) * E], mx["mask"]["size"], mx["scale"])
        heads.append(o * gate[:, a:a + 1])
    return np.concatenate(heads, axis=1) @ W[pre + "o"].T


def token_shift(h, mu):
    """h + (previous h - h) * mu, the token before the first one being zero."""
    prev = np.concatenate([np.zeros_like(h[:1]), h[:-1]], axis=0)
    return h + (prev - h) * mu


def wkv_recurrence(r, k, v, w, u):
    """One head, [tokens, dim] each (u: [dim]): o_t = (S + diag(u) k v^T)^T r, then S = diag(w) S + k v^T."""
    S = np.zeros((k.shape[1], v.shape[1]), k.dtype)
    out = np.zeros_like(v)
    for t in range(k.shape[0]):
        kv = np.outer(k[t], v[t])
        out[t] = (S + u[:, None] * kv).T @ r[t]
        S = w[t][:, None] * S + kv
    return out


def silu(z):
    return z * sigmoid(z)


def wkv_mixer(h, W, pre, mx, eps):
    H, D = mx["heads"], mx["dim"]
    mix = {c: token_shift(h, W[pre + "mu." + c]) for c in "rkvgw"}
    r, k, v = (mix[c] @ W[pre + c].T for c in "rkv")
    gate = silu(mix["g"] @ W[pre + "g"].T)
    w = np.exp(-np.exp(np.tanh(mix["w"] @ W[pre + "w1"].T) @ W[pre + "w2"].T + W[pre + "w0"]))
    u = W[pre + "u"]
    heads = []
    for a in range(H):
        c = slice(a * D, (a + 1) * D)
        heads.append(rms_unit(wkv_recurrence(r[:, c], k[:, c], v[:, c], w[:, c], u[a]), eps))
    return (np.concatenate(heads, axis=1) * W[pre + "norm"] * gate) @ W[pre + "o"].T


def relu_glu(h, W, pre):
    return (np.maximum(h @ W[pre + "gate"].T, 0.0) * (h @ W[pre + "up"].T)) @ W[pre + "down"].T


MIXERS = {"attention": attention_mixer, "wkv": wkv_mixer}


def layer(x, W, i, spec, eps):
    pre = f"l{i}."
    y = MIXERS[spec["type"]](scalar_norm(x, W[pre + "norm1"], eps), W, pre + "mix.", spec["mixer"], eps)
    x = x + scalar_norm(y, W[pre + "norm1b"], eps)
    if spec.get("mlp"):
        y = relu_glu(scalar_norm(x, W[pre + "norm2"], eps), W, pre + "mlp.")
        x = x + scalar_norm(y, W[pre + "norm2b"], eps)
    return x


def layer_runs(cfg):
    """[(layer index, whether a pass of the loop starts right before it)] in execution order."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return ([(i, False) for i in range(a)] + [(i, i == a) for _ in range(loop["times"]) for i in range(a, b)] +
            [(i, False) for i in range(b, n)])


def forward(cfg, W, tokens, dtype=np.float64, want_layers=False):
    """logits [tokens, vocab] of one sequence; with ``want_layers`` also the residual after every layer run."""
    W = {k: np.asarray(a, dtype) for k, a in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)]
    x0, states = x, []
    for i, pass_start in layer_runs(cfg):
        if pass_start:
            x = np.concatenate([x, x0], axis=1) @ W["loop.in"].T
        x = layer(x, W, i, cfg["layers"][i], eps)
        states.append(x)
    logits = (scalar_norm(x, W["final.norm"], eps) @ W["head"].T) * cfg["logit_scale"]
    return (logits, np.stack(states)) if want_layers else logits


def greedy(cfg, W, prompt, count):
    """prompt + ``count`` greedily chosen ids, recomputing the whole sequence for every token."""
    toks = list(prompt)
    for _ in range(count):
        toks.append(int(np.argmax(forward(cfg, W, toks)[-1])))
    return toks
