"""Command line.

    python -m nanochat_b200 generate --model DIR --prompt 1,2,3 [--prompt ...] [--max-new-tokens N] [--temperature T] ...
    python -m nanochat_b200 trace --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N   (steps on standard input)
    python -m nanochat_b200 models

The model class follows from DIR/config.json (registry.py). Prompts and outputs are token ids: tokenising is outside this
package. bin/trace_run is the trace command as a program."""

import argparse
import json
import sys

DTYPE_REFUSED = 3


def parser() -> argparse.ArgumentParser:
    ap = argparse.ArgumentParser(prog="python -m nanochat_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    gen = sub.add_parser("generate", help="continue prompts of token ids, one JSON line per prompt in completion order")
    gen.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    gen.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    gen.add_argument("--prompt", action="append", default=[], help="token ids with commas between them; repeat for more prompts")
    gen.add_argument("--max-new-tokens", type=int, default=32)
    gen.add_argument("--temperature", type=float, default=0.0)
    gen.add_argument("--top-p", type=float, default=1.0)
    gen.add_argument("--seed", type=int, default=0, help="seed of the first prompt; the others count up from it")
    gen.add_argument("--end-token", type=int, default=-1, help="token that ends a continuation (-1: none)")
    gen.add_argument("--slots", type=int, default=8, help="sequences decoded together")
    gen.add_argument("--max-len", type=int, default=0, help="positions per slot (0: what the longest request needs)")
    trace = sub.add_parser("trace", help="replay steps of given tokens from standard input and write the wanted logits")
    trace.add_argument("--model", required=True)
    trace.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    trace.add_argument("--out", required=True, help="folder for <step>.f32")
    trace.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    trace.add_argument("--slots", type=int, default=4, help="requests that can be live together")
    sub.add_parser("models", help="the registered architectures")
    return ap


def main(argv: "list[str] | None" = None) -> int:
    args = parser().parse_args(argv)
    import torch

    from . import registry

    if args.command == "models":
        for name, arch in sorted(registry.ARCHITECTURES.items()):
            print(name, *(str(d).removeprefix("torch.") for d in arch.dtypes))
        return 0
    dtype = getattr(torch, args.dtype)
    try:
        if args.command == "trace":
            from .trace import replay

            decoder = registry.load_decoder(args.model, args.slots, max(args.max_tokens, 1), dtype)
            replay(decoder, sys.stdin, args.out, sys.stdout)
            return 0
        from .serving import NativeDecoder, Request

        prompts = [[int(t) for t in p.split(",")] for p in args.prompt]
        if not prompts:
            return 0
        need = max(map(len, prompts)) - 1 + args.max_new_tokens
        decoder = registry.load_decoder(args.model, min(args.slots, len(prompts)), args.max_len or need, dtype)
    except registry.UnsupportedDtype as e:
        print(e, file=sys.stderr)
        return DTYPE_REFUSED
    requests = [Request(input_ids=p, max_new_tokens=args.max_new_tokens, temperature=args.temperature, top_p=args.top_p,
                        seed=args.seed + i) for i, p in enumerate(prompts)]
    for index, tokens in NativeDecoder(decoder, end_token=args.end_token).generate(requests):
        print(json.dumps({"prompt": index, "tokens": tokens}), flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
