"""Command line: `python -m ytensor_b200 models | generate | trace`.

    python -m ytensor_b200 generate --model DIR --tokens 1,2,3 --steps 32 [--top-k 20 --seed 42] [--dtype float32]

Token ids in and out (tokenizers stay on the host side of the reference)."""
from __future__ import annotations

import argparse
import sys


def main(argv=None) -> int:
    argv = list(sys.argv[1:] if argv is None else argv)
    if argv and argv[0] == "trace":
        from .trace import main as trace_main
        return trace_main(argv[1:])
    ap = argparse.ArgumentParser(prog="python -m ytensor_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    sub.add_parser("models", help="list the registered models")
    sub.add_parser("trace", help="replay a trace of token ids (see --help of the subcommand)", add_help=False)
    g = sub.add_parser("generate", help="generate tokens")
    g.add_argument("--model", required=True, help="folder with config.json and the weights")
    g.add_argument("--tokens", required=True, help="prompt: comma-separated token ids; several prompts of one length: ';'")
    g.add_argument("--steps", type=int, default=32)
    g.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    g.add_argument("--max-tokens", type=int, default=0, help="longest sequence (default: prompt and steps)")
    g.add_argument("--top-k", type=int, default=0, help="sample among the k most probable tokens (default: greedy)")
    g.add_argument("--seed", type=int, default=42)
    a = ap.parse_args(argv)
    from .registry import MODELS, load_model
    if a.command == "models":
        for m in MODELS.values():
            print(m.name, *m.dtypes)
        return 0
    prompts = [[int(t) for t in p.split(",")] for p in a.tokens.split(";")]
    if len({len(p) for p in prompts}) != 1:
        ap.error("the prompts of one call must have the same length")
    import torch
    model = load_model(a.model, dtype=a.dtype, batch=len(prompts), build=True,
                       max_tokens=a.max_tokens or len(prompts[0]) + a.steps)
    ids = torch.tensor(prompts, dtype=torch.int32, device="cuda")
    out = model.generate_topk(ids, a.steps, k=a.top_k, seed=a.seed) if a.top_k else model.generate_greedy(ids, a.steps)
    for row in out.cpu().tolist():
        print(",".join(map(str, row)))
    model.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
