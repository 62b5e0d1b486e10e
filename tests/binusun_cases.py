"""Small Binusun configurations and helpers shared by the CPU and GPU tests."""
import numpy as np

from caten_b200 import synthetic as S
from caten_b200.safetensors import bf16_to_f32

SCALING = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 256}

# name -> (configuration, rank of the decay projection); head sizes that are and are not multiples of 16, grouped and
# single key/value heads, windows from one token up, loops at the start, in the middle, over everything and none
CASES = {
    "attention": (S.binusun_config(96, 131, "A", 80, 4, 2, 32, 32, 9, 1, 16, 32, scale=0.4), 8),
    "wkv": (S.binusun_config(64, 100, "w", 64, 1, 1, 16, 16, 4, 2, 24, 16), 200),
    "mixed": (S.binusun_config(160, 203, "wAaW", 96, 6, 2, 40, 24, 21, 3, 16, 12, rot_base=500.0, scaling=SCALING, loop=(1, 3, 2), logit_scale=1.5), 11),
    "loop_all": (S.binusun_config(72, 97, "Aw", 40, 3, 3, 20, 48, 33, 2, 40, 20, loop=(0, 2, 3), eps=1e-3), 16),
    "loop_once": (S.binusun_config(256, 64, "aWA", 192, 8, 1, 64, 64, 70, 2, 64, 64, scaling=SCALING, loop=(2, 3, 1), logit_scale=0.5), 70),
    "window_one": (S.binusun_config(128, 80, "aA", 64, 2, 1, 128, 96, 1, 1, 16, 2), 4),
    "wide_heads": (S.binusun_config(64, 75, "aW", 64, 2, 1, 136, 200, 40, 1, 136, 100), 3),
}
_cache = {}


def case(name):
    """(configuration, bf16 tensors, fp32 weights for the oracle)"""
    if name not in _cache:
        cfg, rank = CASES[name]
        t = S.synth_binusun(cfg, seed=sum(map(ord, name)), low_rank=rank)
        _cache[name] = cfg, t, {k: bf16_to_f32(v) for k, v in t.items()}
    return _cache[name]


def tokens(name, count, seed=0):
    return np.random.Generator(np.random.PCG64(seed)).integers(0, CASES[name][0]["vocab"], size=count, dtype=np.int64)


def rel_rms(got, want):
    """Root mean square of the difference over that of ``want`` (mean over the vocabulary taken off), per row."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.sqrt(want.var(axis=-1).mean())
