"""Command line: greedy generation from token ids.

    python -m cera_b200 generate --model DIR_OR_GGUF --tokens 1,2,3 --n 16 [--dtype bfloat16|float32] [--max-seq-len N]
"""
import argparse

import numpy as np

from .registry import load_model


def generate(a):
    prompt = [int(t) for t in a.tokens.split(",")]
    kw = {"dtype": a.dtype} if a.dtype else {}
    model = load_model(a.model, max_seq_len=a.max_seq_len or len(prompt) + a.n, **kw)
    out = [int(np.argmax(model.forward_prefill(prompt, 0)))] if a.n else []
    if a.n > 1:
        rest, _ = model.generate_greedy(out[0], len(prompt), a.n - 1)
        out += [int(t) for t in rest]
    model.close()
    print(" ".join(map(str, out)))


def main():
    ap = argparse.ArgumentParser(prog="cera_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="greedy tokens after a prompt of token ids")
    g.add_argument("--model", required=True, help="folder with config.json and model.safetensors, or a GGUF file")
    g.add_argument("--tokens", required=True, help="prompt token ids, comma-separated")
    g.add_argument("--n", type=int, default=16, help="tokens to generate")
    g.add_argument("--dtype", choices=["bfloat16", "float32"], help="compute type of a folder model (default bfloat16)")
    g.add_argument("--max-seq-len", type=int)
    g.set_defaults(run=generate)
    a = ap.parse_args()
    a.run(a)


if __name__ == "__main__":
    main()
