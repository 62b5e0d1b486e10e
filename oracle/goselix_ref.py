"""Plain statement of the Goselix decoder in numpy: whole sequences, no cache, no state carried between
calls, loops over tokens, heads and experts.  Test infrastructure; shares no code with the package.

``cfg`` is the parsed config.json of a model, ``W`` maps tensor names to arrays.  Every function works in
the dtype of its inputs (float64 unless a caller passes something else).
"""
from __future__ import annotations

import math

import numpy as np


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, g, eps):
    """RMS norm with one gain per coordinate."""
    return rms_unit(x, eps) * g


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rotate_halves(x, dims, base, first_position=0):
    """x [tokens, dim]: coordinate i < dims / 2 turns with coordinate i + dims / 2 by position * base^(-2i / dims);
    the coordinates from ``dims`` on stay."""
    y, half = x.copy(), dims // 2
    for t in range(x.shape[0]):
        for i in range(half):
            a = (first_position + t) * base ** (-2.0 * i / dims)
            c, s = math.cos(a), math.sin(a)
            u, v = x[t, i], x[t, half + i]
            y[t, i], y[t, half + i] = u * c - v * s, v * c + u * s
    return y


def causal_attention(q, k, v, scale):
    """One head: query i sees the keys up to i; ordinary softmax."""
    out = np.zeros((q.shape[0], v.shape[1]), q.dtype)
    for i in range(q.shape[0]):
        s = (k[:i + 1] @ q[i]) * scale
        p = np.exp(s - s.max())
        out[i] = (p / p.sum()) @ v[:i + 1]
    return out


def latent_attention_mixer(h, W, pre, mx, eps):
    """Queries, keys and values of all heads come from two normed latents; a rotated key part is common to the heads."""
    H, D, P, E, K = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    base = mx["rot"]["base"]
    cq = rms_norm(h @ W[pre + "dq"].T, W[pre + "dq.norm"], eps)
    q = cq @ W[pre + "uq"].T
    down = h @ W[pre + "dkv"].T
    c = rms_norm(down[:, :K], W[pre + "dkv.norm"], eps)
    shared = rotate_halves(down[:, K:], P, base)
    heads = []
    for a in range(H):
        qa = q[:, a * (D + P):(a + 1) * (D + P)]
        qa = np.concatenate([qa[:, :D], rotate_halves(qa[:, D:], P, base)], axis=1)
        ka = np.concatenate([c @ W[pre + "uk"][a * D:(a + 1) * D].T, shared], axis=1)
        heads.append(causal_attention(qa, ka, c @ W[pre + "uv"][a * E:(a + 1) * E].T, mx["scale"]))
    return np.concatenate(heads, axis=1) @ W[pre + "o"].T


def retention_recurrence(q, k, v, decay):
    """One head: S = decay S + k v^T, o = S^T q, from S = 0."""
    S = np.zeros((k.shape[1], v.shape[1]), k.dtype)
    out = np.zeros_like(v)
    for t in range(k.shape[0]):
        S = decay * S + np.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out


def retention_mixer(h, W, pre, mx, eps):
    H, D, E, rot = mx["heads"], mx["dim"], mx["vdim"], mx["rot"]
    q, k, v = h @ W[pre + "q"].T, h @ W[pre + "k"].T, h @ W[pre + "v"].T
    heads = []
    for a in range(H):
        qa = rotate_halves(q[:, a * D:(a + 1) * D], rot["dims"], rot["base"])
        ka = rotate_halves(k[:, a * D:(a + 1) * D], rot["dims"], rot["base"]) * D ** -0.5
        heads.append(rms_unit(retention_recurrence(qa, ka, v[:, a * E:(a + 1) * E], mx["decay"][a]), eps))
    return (np.concatenate(heads, axis=1) * silu(h @ W[pre + "g"].T)) @ W[pre + "o"].T


def silu_glu(h, W, pre):
    return (silu(h @ W[pre + "gate"].T) * (h @ W[pre + "up"].T)) @ W[pre + "down"].T


def route(h, W, pre, top):
    """[(expert, weight)] per token: the ``top`` largest sigmoid scores, which are the weights as they are."""
    s = sigmoid(h @ W[pre + "router"].T)
    return [[(int(e), s[t, e]) for e in np.argsort(-s[t], kind="stable")[:top]] for t in range(h.shape[0])]


def expert_mixture(h, W, pre, spec):
    """The weight scales what goes into an expert."""
    out = np.zeros_like(h)
    for t, chosen in enumerate(route(h, W, pre, spec["router"]["top"])):
        for e, w in chosen:
            out[t] += silu_glu(w * h[t:t + 1], W, f"{pre}e{e}.")[0]
    return out


MIXERS = {"latent_attention": latent_attention_mixer, "retention": retention_mixer}


def feed_forward(h, W, pre, spec):
    return silu_glu(h, W, pre) if spec["kind"] == "dense" else expert_mixture(h, W, pre, spec)


def layer(x, W, i, spec, eps):
    """Mixer and feed-forward side by side, each with its own norm of the same stream."""
    pre = f"l{i}."
    y = MIXERS[spec["type"]](rms_norm(x, W[pre + "norm1"], eps), W, pre + "mix.", spec["mixer"], eps)
    if spec.get("mlp"):
        y = y + feed_forward(rms_norm(x, W[pre + "norm2"], eps), W, pre + "mlp.", spec["mlp"])
    return x + y


def layer_runs(cfg):
    """[(layer index, number of the loop pass that starts right before it, or None)] in execution order."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return ([(i, None) for i in range(a)] + [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)] +
            [(i, None) for i in range(b, n)])


def forward(cfg, W, tokens, dtype=np.float64, want_layers=False):
    """logits [tokens, vocab] of one sequence; with ``want_layers`` also the residual after every layer run."""
    W = {k: np.asarray(a, dtype) for k, a in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)]
    x0, states = x, []
    for i, t in layer_runs(cfg):
        if t is not None:
            x = (x + x0 if t > 0 else x) + W["loop.step"][t]
        x = layer(x, W, i, cfg["layers"][i], eps)
        states.append(x)
    logits = rms_norm(x, W["final.norm"], eps) @ W["head"].T
    return (logits, np.stack(states)) if want_layers else logits


def greedy(cfg, W, prompt, count):
    """prompt + ``count`` greedily chosen ids, recomputing the whole sequence for every token."""
    toks = list(prompt)
    for _ in range(count):
        toks.append(int(np.argmax(forward(cfg, W, toks)[-1])))
    return toks
