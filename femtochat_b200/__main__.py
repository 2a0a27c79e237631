"""Command line: `python -m femtochat_b200 generate --model DIR --tokens 5,17,3` and `... trace` (the trace runner)."""
from __future__ import annotations

import argparse
import sys


def generate_main(argv) -> int:
    ap = argparse.ArgumentParser(prog="femtochat_b200 generate", description="Continue a prompt of token ids with a model from a folder.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--tokens", required=True, help="prompt: token ids separated by commas")
    ap.add_argument("--max-new-tokens", type=int, default=20)
    ap.add_argument("--temperature", type=float, default=0.8, help="0 = greedy")
    ap.add_argument("--top-k", type=int, default=40)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    a = ap.parse_args(argv)
    import torch
    from .generation import generate
    from .models import load_model
    model = load_model(a.model, compute_type=a.dtype)
    tokens = [int(t) for t in a.tokens.split(",") if t.strip()]
    out = generate(model, tokens, max_new_tokens=a.max_new_tokens, temperature=a.temperature, top_k=a.top_k,
                   generator=torch.Generator().manual_seed(a.seed))
    print(",".join(str(t) for t in out[len(tokens):]))
    return 0


def main() -> int:
    from . import trace
    commands = {"generate": generate_main, "trace": trace.main}
    if len(sys.argv) < 2 or sys.argv[1] not in commands:
        print(f"usage: python -m femtochat_b200 {{{','.join(commands)}}} ...", file=sys.stderr)
        return 2
    return commands[sys.argv[1]](sys.argv[2:])


if __name__ == "__main__":
    sys.exit(main())
