"""Small Goselix configurations and helpers shared by the CPU and GPU tests."""
import numpy as np

from caten_b200 import synthetic as S
from caten_b200.safetensors import bf16_to_f32, f32_to_bf16

# name -> configuration; head sizes and ranks that are and are not multiples of 16, all kinds of feed-forward, several experts
# per token, loops at the start, in the middle, over everything and none
CASES = {
    #                           width vocab order      ff  H  D   P   E   Qr  Kr   ret: H  D   E   rot
    "latent": S.goselix_config(96, 131, "l-", 16, 3, 20, 12, 24, 40, 33, 1, 16, 16, 16, scale=0.4, rot_base=500.0),
    "retention": S.goselix_config(72, 100, "r-", 16, 1, 16, 16, 16, 16, 16, 4, 24, 40, 16, decay=(1.0, 0.99, 0.7, 0.25), ret_base=300.0),
    "dense": S.goselix_config(160, 203, "ldrd", 80, 5, 32, 16, 48, 72, 64, 2, 32, 64, 32, eps=1e-3),
    "experts": S.goselix_config(128, 90, "lmrm", 16, 2, 16, 8, 16, 24, 40, 2, 16, 32, 8, experts=5, top=3, expert_ff=40),
    "experts_many": S.goselix_config(64, 77, "rm", 16, 1, 16, 16, 16, 16, 16, 1, 16, 16, 0, experts=70, top=2, expert_ff=16),
    "mixed": S.goselix_config(112, 151, "rdlml-rm", 56, 4, 24, 10, 16, 48, 80, 3, 20, 36, 12, experts=4, top=1, expert_ff=24, loop=(1, 3, 3)),
    "loop_all": S.goselix_config(64, 97, "lmrd", 40, 2, 32, 32, 32, 32, 32, 2, 16, 16, 16, experts=3, top=2, expert_ff=16, loop=(0, 2, 2)),
    "loop_once": S.goselix_config(256, 64, "r-ld", 192, 8, 64, 32, 64, 128, 256, 4, 64, 128, 64, loop=(1, 2, 1)),
    "many_heads": S.goselix_config(64, 70, "ld", 24, 40, 16, 6, 16, 30, 130, 1, 16, 16, 16),
    "wide": S.goselix_config(64, 75, "l-rd", 64, 2, 100, 40, 140, 70, 600, 1, 136, 300, 100),
    "rank512": S.goselix_config(80, 61, "l-", 64, 18, 16, 64, 32, 48, 512, 1, 16, 16, 16),
}
_cache = {}


def weights(t):
    """fp32 weights for the oracle"""
    return {k: bf16_to_f32(v) for k, v in t.items()}


def case(name):
    """(configuration, bf16 tensors, fp32 weights for the oracle)"""
    if name not in _cache:
        t = S.synth_goselix(CASES[name], seed=sum(map(ord, name)))
        _cache[name] = CASES[name], t, weights(t)
    return _cache[name]


def has_experts(name):
    return any(l["mlp"] and l["mlp"]["kind"] == "moe" for l in CASES[name]["layers"])


def tokens(name, count, seed=0):
    return np.random.Generator(np.random.PCG64(seed)).integers(0, CASES[name]["vocab"], size=count, dtype=np.int64)


def rel_rms(got, want):
    """Root mean square of the difference over that of ``want`` (mean over the vocabulary taken off), per row."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.sqrt(want.var(axis=-1).mean())


def far_config(kind, loop=None):
    """One layer, one mixer, sizes that leave room for :func:`plant`."""
    return S.goselix_config(64, 40, "l-" if kind == "latent" else "r-", 16, 3, 32, 16, 32, 32, 48, 2, 32, 32, 16, decay=(0.9999, 0.999), scale=1.0, loop=loop)


def plant(cfg, kind, seed=0):
    """Weights with which token 1 asks for token 0: their embeddings turn a query and a key to one direction that nothing else
    uses, so that the score (or the product with the state) of that pair stands out however far the two are apart, and what
    token 0 brings has a value of its own."""
    t = S.synth_goselix(cfg, seed=seed)
    w, m = weights(t), cfg["layers"][0]["mixer"]
    width, H, D = cfg["width"], m["heads"], m["dim"]
    asks, has = np.zeros(width, np.float32), np.zeros(width, np.float32)
    asks[0], has[1] = 8.0, 8.0            # unit root mean square in 64 dims
    w["embed"][:, :2] = 0.0
    w["embed"][1], w["embed"][0] = asks, has
    mix = "l0.mix."
    w["l0.norm1"][:] = 1.0
    if kind == "latent":
        P, E = m["rot_dim"], m["vdim"]
        for n in ("dq", "dkv"):
            w[mix + n] *= 0.3
        w[mix + "dq.norm"][:] = w[mix + "dkv.norm"][:] = 1.0
        w[mix + "dq"][0, 0], w[mix + "dkv"][0, 1] = 4.0, 4.0     # latent coordinate 0
        for h in range(H):
            w[mix + "uq"][h * (D + P):(h + 1) * (D + P), 0] = 0.0
            w[mix + "uk"][h * D:(h + 1) * D, 0] = 0.0
            w[mix + "uq"][h * (D + P), 0] = w[mix + "uk"][h * D, 0] = 1.0
            w[mix + "uv"][h * E:(h + 1) * E, 0] = 1.0
    else:
        for n in ("q", "k"):
            w[mix + n] *= 0.02
        for h in range(H):
            w[mix + "q"][h * D + D - 1, 0] = w[mix + "k"][h * D + D - 1, 1] = 1.0   # a dim that does not turn
    return {k: f32_to_bf16(v) for k, v in w.items()}
