"""Command line: generate token ids (or text, with a GGUF file's tokenizer) from a stored model.

    python -m caten_b200.generate --model DIR_OR_GGUF (--ids 5,17,3 | --prompt TEXT) [--max-length N]
                                  [--precision fp32|bf16|bf16x3] [--temperature T --top-k K --seed S]
"""
from __future__ import annotations

import argparse

from .model import generate
from .registry import load_model
from .runtime import B200Runtime


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="caten_b200.generate")
    ap.add_argument("--model", required=True, help="a GGUF file, or a folder with config.json and model.safetensors")
    src = ap.add_mutually_exclusive_group(required=True)
    src.add_argument("--ids", help="prompt as comma-separated token ids")
    src.add_argument("--prompt", help="prompt as text (GGUF models, which bring a tokenizer)")
    ap.add_argument("--max-length", type=int, default=32, help="tokens to generate")
    ap.add_argument("--precision", default="bf16x3", choices=["fp32", "bf16", "bf16x3"])
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--device", type=int, default=0)
    args = ap.parse_args(argv)
    tok = None
    if args.prompt is not None:
        from .bpe import gguf_to_bpe_tokenizer
        from .gguf import load_gguf
        tok = gguf_to_bpe_tokenizer(load_gguf(args.model))
        ids = tok.encode(args.prompt)
    else:
        ids = [int(x) for x in args.ids.split(",")]
    with B200Runtime(args.device) as rt:
        m = load_model(args.model, rt, max_seq_len=len(ids) + args.max_length, batch=1, precision=args.precision)
        out = generate(m, [ids], args.max_length, args.temperature, args.top_k, args.seed)[0].tolist()
        m.close()
    print(tok.decode(out) if tok is not None else ",".join(str(i) for i in out))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
