"""Seeded synthetic GPT-2 state dicts and prompts.

Pre-trained GPT-2 GGUF files (apps/gpt2/gpt2.lisp:50 downloads them) are not available offline,
so every configuration is generated from ``numpy.random.Generator(PCG64(seed))`` with the shapes
and value distributions the benchmark configurations state.  Quantised weights are generated
directly in packed GGUF block form (codes + fp16 scale), so their dequantised values are exact.

State-dict keys are the reference's after `remap-state-dict-keys` (apps/gpt2/gpt2.lisp:52-80).
A quantised entry is a :class:`Packed` (raw GGUF block bytes, ggml type id, logical shape).
"""
from __future__ import annotations

from dataclasses import dataclass

import numpy as np

GGML_F32, GGML_F16, GGML_Q4_0, GGML_Q4_1, GGML_Q5_0, GGML_Q5_1, GGML_Q8_0 = 0, 1, 2, 3, 6, 7, 8
BLOCK_BYTES = {GGML_Q4_0: 18, GGML_Q4_1: 20, GGML_Q5_0: 22, GGML_Q5_1: 24, GGML_Q8_0: 34}
TYPE_IDS = {"f32": GGML_F32, "f16": GGML_F16, "q4_0": GGML_Q4_0, "q4_1": GGML_Q4_1, "q5_0": GGML_Q5_0, "q5_1": GGML_Q5_1,
            "q8_0": GGML_Q8_0}


@dataclass(frozen=True)
class GPT2Params:
    """Model sizes of apps/gpt2/gpt2.lisp:36-41 (head dim is 64 for all of them)."""
    n_layers: int
    n_heads: int
    dim: int
    vocab_size: int = 50257
    norm_eps: float = 1e-5


GPT2_SIZES = {
    "gpt2": GPT2Params(12, 12, 768),
    "gpt2-medium": GPT2Params(24, 16, 1024),
    "gpt2-large": GPT2Params(36, 20, 1280),
    "gpt2-xl": GPT2Params(48, 25, 1600),
}


@dataclass
class Packed:
    """A weight matrix [rows, cols] kept as raw GGUF blocks (row-major, cols/32 blocks per row)."""
    ggml_type: int
    rows: int
    cols: int
    data: np.ndarray  # uint8, flat

    @property
    def shape(self):
        return (self.rows, self.cols)


def pack_q8_0(codes: np.ndarray, scales: np.ndarray) -> np.ndarray:
    """codes int8 [..., 32], scales float16 [...] -> uint8 [..., 34] (scale first, then 32 int8)."""
    nb = int(np.prod(scales.shape))
    out = np.empty((nb, 34), np.uint8)
    out[:, 0:2] = np.ascontiguousarray(scales, dtype="<f2").reshape(nb, 1).view(np.uint8)
    out[:, 2:] = np.ascontiguousarray(codes, dtype=np.int8).reshape(nb, 32).view(np.uint8)
    return out.reshape(-1)


def pack_q4_0(codes: np.ndarray, scales: np.ndarray) -> np.ndarray:
    """codes uint8 in [0,15] [..., 32], scales float16 [...] -> uint8 [..., 18].

    Byte j of a block holds element j in its low nibble and element j+16 in its high nibble."""
    nb = int(np.prod(scales.shape))
    c = np.ascontiguousarray(codes, dtype=np.uint8).reshape(nb, 32)
    out = np.empty((nb, 18), np.uint8)
    out[:, 0:2] = np.ascontiguousarray(scales, dtype="<f2").reshape(nb, 1).view(np.uint8)
    out[:, 2:] = (c[:, :16] & 0x0F) | (c[:, 16:] << 4)
    return out.reshape(-1)


def _rand_packed(rng: np.random.Generator, rows: int, cols: int, wtype: str, std: float = 0.02) -> Packed:
    assert cols % 32 == 0
    nb = rows * (cols // 32)
    if wtype == "q8_0":
        # 32 int8 uniform in [-127, 127]; scale = |N(0, 0.02)| / 127
        codes = rng.integers(-127, 128, size=(nb, 32), dtype=np.int8)
        scales = (np.abs(rng.standard_normal(nb, dtype=np.float32)) * np.float32(std / 127)).astype(np.float16)
        return Packed(GGML_Q8_0, rows, cols, pack_q8_0(codes, scales))
    if wtype == "q4_0":
        # 32 4-bit codes uniform in [0, 15] (offset 8); scale = |N(0, 0.02)| / 8.  A uniform byte
        # is two independent uniform nibbles, so the quant bytes are drawn directly.
        out = np.empty((nb, 18), np.uint8)
        out[:, 2:] = rng.integers(0, 256, size=(nb, 16), dtype=np.uint8)
        scales = (np.abs(rng.standard_normal(nb, dtype=np.float32)) * np.float32(std / 8)).astype("<f2")
        out[:, 0:2] = scales.reshape(nb, 1).view(np.uint8)
        return Packed(GGML_Q4_0, rows, cols, out.reshape(-1))
    if wtype in ("q4_1", "q5_0", "q5_1"):
        # uniform code bytes (and fifth bits); scale = |N(0, std)| / half the code range; the _1
        # formats get a minimum that centres the codes: m = -(range / 2) * d + N(0, std / 16)
        t = TYPE_IDS[wtype]
        levels = 16 if wtype == "q4_1" else 32
        out = rng.integers(0, 256, size=(nb, BLOCK_BYTES[t]), dtype=np.uint8)
        d = (np.abs(rng.standard_normal(nb, dtype=np.float32)) * np.float32(std / (levels / 2))).astype("<f2")
        out[:, 0:2] = d.reshape(nb, 1).view(np.uint8)
        if wtype != "q5_0":
            m = (-(levels / 2) * d.astype(np.float32) + rng.standard_normal(nb, dtype=np.float32) * np.float32(std / 16)).astype("<f2")
            out[:, 2:4] = m.reshape(nb, 1).view(np.uint8)
        return Packed(t, rows, cols, out.reshape(-1))
    raise ValueError(wtype)


def synth_state_dict(p: GPT2Params, wtype: str = "f32", seed: int = 0, max_seq_len: int = 1024,
                     trivial_affine: bool = True, weight_std: float = 0.02) -> dict:
    """Draw order (fixed): wte, wpe, then per layer c_attn, attn.c_proj, mlp.c_fc, mlp.c_proj
    (weight, then bias/affine extras when ``trivial_affine`` is False), then lm_head.

    wtype "f32": every matrix ~ N(0, 0.02).  "q8_0"/"q4_0"/"q4_1"/"q5_0"/"q5_1": the five kinds of Linear weight are
    packed blocks; embeddings, LayerNorm parameters and biases stay fp32.
    ``trivial_affine``: biases 0, LayerNorm gamma 1 / beta 0 (the benchmark configurations);
    False draws them at random so tests exercise those terms.  ``weight_std`` scales the fp32
    matrices and the quantisation scales (0.02 in the benchmark configurations; tests use a
    larger value so that sequences and logits differ visibly)."""
    rng = np.random.Generator(np.random.PCG64(seed))
    d, L, V = p.dim, p.n_layers, p.vocab_size

    def normal(*shape):
        return (rng.standard_normal(shape, dtype=np.float32) * np.float32(weight_std))

    def lin(rows, cols):
        return normal(rows, cols) if wtype == "f32" else _rand_packed(rng, rows, cols, wtype, weight_std)

    def vec(n, base):
        if trivial_affine:
            return np.full(n, base, np.float32)
        return (np.float32(base) + rng.standard_normal(n, dtype=np.float32) * np.float32(0.1))

    sd = {"wte.weight": normal(V, d), "wpe.weight": normal(max_seq_len, d)}
    for l in range(L):
        pre = f"h.{l}."
        sd[pre + "ln_1.affine"] = vec(d, 1.0)
        sd[pre + "ln_1.bias"] = vec(d, 0.0)
        sd[pre + "attn.c_attn.weight"] = lin(3 * d, d)
        sd[pre + "attn.c_attn.bias"] = vec(3 * d, 0.0)
        sd[pre + "attn.c_proj.weight"] = lin(d, d)
        sd[pre + "attn.c_proj.bias"] = vec(d, 0.0)
        sd[pre + "ln_2.affine"] = vec(d, 1.0)
        sd[pre + "ln_2.bias"] = vec(d, 0.0)
        sd[pre + "mlp.c_fc.weight"] = lin(4 * d, d)
        sd[pre + "mlp.c_fc.bias"] = vec(4 * d, 0.0)
        sd[pre + "mlp.c_proj.weight"] = lin(d, 4 * d)
        sd[pre + "mlp.c_proj.bias"] = vec(d, 0.0)
    sd["ln_f.affine"] = vec(d, 1.0)
    sd["ln_f.bias"] = vec(d, 0.0)
    sd["lm_head.weight"] = lin(V, d)
    return sd


def binusun_config(width: int, vocab: int, order: str, ff: int, heads: int, kv_heads: int, dim: int, vdim: int, window: int, wkv_heads: int, wkv_dim: int,
                   rot_dims: int, rot_base: float = 10000.0, scaling: dict | None = None, scale: float | None = None, loop: tuple | None = None,
                   eps: float = 1e-5, logit_scale: float = 1.0) -> dict:
    """A Binusun configuration (the content of config.json).  ``order``: one letter per layer, "a" attention or "w"
    time mixing; an upper-case letter adds a feed-forward of width ``ff``.  ``loop``: (start, stop, times)."""
    att = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "scale": dim ** -0.5 if scale is None else scale,
           "rot": {"base": rot_base, "dims": rot_dims, "scaling": scaling}}
    mix = {"heads": wkv_heads, "dim": wkv_dim}
    layers = [{"type": "attention" if c in "aA" else "wkv", "mixer": dict(att) if c in "aA" else dict(mix),
               "mlp": {"kind": "dense", "ff": ff} if c.isupper() else None} for c in order]
    return {"architecture": "Binusun", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "loop": {"start": loop[0], "stop": loop[1], "times": loop[2]} if loop else None}


def synth_binusun(cfg: dict, seed: int = 0, low_rank: int = 16) -> dict:
    """Random weights of a Binusun configuration: tensor name -> bf16 bit patterns (uint16).  Matrices ~ N(0, 1 / in),
    so that projections of a normed row have unit scale; norm gains around 1; the decays spread over (0, 1)."""
    from .safetensors import f32_to_bf16
    rng = np.random.Generator(np.random.PCG64(seed))
    width, vocab, t = cfg["width"], cfg["vocab"], {}

    def mat(name, rows, cols):
        t[name] = f32_to_bf16(rng.standard_normal((rows, cols), dtype=np.float32) * np.float32(cols ** -0.5))

    def vec(name, shape, mean, std):
        t[name] = f32_to_bf16(np.float32(mean) + rng.standard_normal(shape, dtype=np.float32) * np.float32(std))

    t["embed"] = f32_to_bf16(rng.standard_normal((vocab, width), dtype=np.float32))
    if cfg.get("loop"):
        mat("loop.in", width, 2 * width)
    for i, l in enumerate(cfg["layers"]):
        pre, m = f"l{i}.", l["mixer"]
        mix = pre + "mix."
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if l["mlp"] else ()):
            vec(pre + n, (), 1.0, 0.1)
        if l["type"] == "attention":
            H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, r in (("q", H * D), ("k", G * D), ("v", G * E), ("g", H)):
                mat(mix + n, r, width)
            mat(mix + "o", width, H * E)
        else:
            hd = m["heads"] * m["dim"]
            for c in "rkvgw":
                vec(mix + "mu." + c, (width,), 0.5, 0.25)
            for c in "rkvg":
                mat(mix + c, hd, width)
            mat(mix + "w1", low_rank, width)
            mat(mix + "w2", hd, low_rank)
            vec(mix + "w0", (hd,), -2.0, 1.5)
            vec(mix + "u", (m["heads"], m["dim"]), 0.0, 0.5)
            vec(mix + "norm", (hd,), 1.0, 0.1)
            mat(mix + "o", width, hd)
        if l["mlp"]:
            mat(pre + "mlp.gate", l["mlp"]["ff"], width)
            mat(pre + "mlp.up", l["mlp"]["ff"], width)
            mat(pre + "mlp.down", width, l["mlp"]["ff"])
    vec("final.norm", (), 1.0, 0.1)
    mat("head", vocab, width)
    return t


def goselix_config(width: int, vocab: int, order: str, ff: int, heads: int, dim: int, rot_dim: int, vdim: int, q_rank: int, kv_rank: int, ret_heads: int,
                   ret_dim: int, ret_vdim: int, ret_rot: int, experts: int = 4, top: int = 1, expert_ff: int = 32, rot_base: float = 10000.0,
                   ret_base: float = 10000.0, scale: float | None = None, decay=None, loop: tuple | None = None, eps: float = 1e-5) -> dict:
    """A Goselix configuration (the content of config.json).  ``order``: two letters per layer, "l" latent attention or
    "r" retention, then "d" a dense feed-forward, "m" a mixture of experts or "-" none.  ``loop``: (start, stop, times)."""
    lat = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
           "scale": (dim + rot_dim) ** -0.5 if scale is None else scale, "rot": {"base": rot_base, "dims": rot_dim}}
    ret = {"heads": ret_heads, "dim": ret_dim, "vdim": ret_vdim, "rot": {"base": ret_base, "dims": ret_rot},
           "decay": list(decay) if decay is not None else [1.0 - 2.0 ** (-3 - h % 8) for h in range(ret_heads)]}
    mlp = {"d": {"kind": "dense", "ff": ff}, "m": {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": expert_ff}}, "-": None}
    layers = [{"type": "latent_attention" if a == "l" else "retention", "mixer": dict(lat) if a == "l" else dict(ret), "mlp": mlp[b]}
              for a, b in zip(order[0::2], order[1::2])]
    return {"architecture": "Goselix", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "loop": {"start": loop[0], "stop": loop[1], "times": loop[2]} if loop else None}


def synth_goselix(cfg: dict, seed: int = 0) -> dict:
    """Random weights of a Goselix configuration: tensor name -> bf16 bit patterns (uint16).  Matrices ~ N(0, 1 / in); norm
    gains around 1; router rows large enough that scores spread over (0, 1) and choices are rarely close."""
    from .safetensors import f32_to_bf16
    rng = np.random.Generator(np.random.PCG64(seed))
    width, vocab, t = cfg["width"], cfg["vocab"], {}

    def mat(name, rows, cols, gain=1.0):
        t[name] = f32_to_bf16(rng.standard_normal((rows, cols), dtype=np.float32) * np.float32(gain * cols ** -0.5))

    def vec(name, shape, mean, std):
        t[name] = f32_to_bf16(np.float32(mean) + rng.standard_normal(shape, dtype=np.float32) * np.float32(std))

    def glu(pre, ff):
        mat(pre + "gate", ff, width)
        mat(pre + "up", ff, width)
        mat(pre + "down", width, ff)

    t["embed"] = f32_to_bf16(rng.standard_normal((vocab, width), dtype=np.float32))
    if cfg.get("loop"):
        vec("loop.step", (cfg["loop"]["times"], width), 0.0, 0.5)
    for i, l in enumerate(cfg["layers"]):
        pre, m, mlp = f"l{i}.", l["mixer"], l["mlp"]
        mix = pre + "mix."
        H, D, E = m["heads"], m["dim"], m["vdim"]
        for n in ("norm1", "norm2")[:2 if mlp else 1]:
            vec(pre + n, (width,), 1.0, 0.1)
        if l["type"] == "latent_attention":
            P, Q, K = m["rot_dim"], m["q_rank"], m["kv_rank"]
            mat(mix + "dq", Q, width)
            vec(mix + "dq.norm", (Q,), 1.0, 0.1)
            mat(mix + "uq", H * (D + P), Q)
            mat(mix + "dkv", K + P, width)
            vec(mix + "dkv.norm", (K,), 1.0, 0.1)
            mat(mix + "uk", H * D, K)
            mat(mix + "uv", H * E, K)
        else:
            for c, n in (("q", D), ("k", D), ("v", E), ("g", E)):
                mat(mix + c, H * n, width)
        mat(mix + "o", width, H * E)
        if mlp and mlp["kind"] == "dense":
            glu(pre + "mlp.", mlp["ff"])
        elif mlp:
            mat(pre + "mlp.router", mlp["router"]["experts"], width, 2.0)
            for e in range(mlp["router"]["experts"]):
                glu(f"{pre}mlp.e{e}.", mlp["expert"]["ff"])
    vec("final.norm", (width,), 1.0, 0.1)
    mat("head", vocab, width)
    return t


def synth_prompts(batch: int, length: int, vocab: int, seed: int = 0) -> np.ndarray:
    """[batch, length] int64 token ids uniform in [0, vocab)."""
    rng = np.random.Generator(np.random.PCG64(seed))
    return rng.integers(0, vocab, size=(batch, length), dtype=np.int64)


def synth_relu_gemm(seed: int = 1, M: int = 4096, K: int = 768, N: int = 3072):
    """A [M,K], B [K,N] with entries N(0,1)/sqrt(K) (the `!relu(!matmul)` configuration)."""
    rng = np.random.Generator(np.random.PCG64(seed))
    sc = np.float32(1.0 / np.sqrt(K))
    return (rng.standard_normal((M, K), dtype=np.float32) * sc,
            rng.standard_normal((K, N), dtype=np.float32) * sc)
