"""Command line.

    python -m buddy_mlir_b200 generate --model DIR --tokens 1,2,3 --max-new 32
    python -m buddy_mlir_b200 trace --model DIR --dtype bfloat16 --out DIR --max-tokens N < steps

Token ids in, token ids out (no tokenizer).  DIR holds config.json and model.safetensors of an
architecture in the registry.
"""
import argparse
import sys


def _generate(a):
    from .registry import load_model
    from .session import run_generation
    s = load_model(a.model, dtype=a.dtype, max_len=a.max_len)
    prompt = [int(t) for t in a.tokens.replace(",", " ").split()]
    stop = [int(t) for t in a.stop.replace(",", " ").split()]
    ids, rate = run_generation(s, prompt, len(prompt) + a.max_new, stop_token_ids=stop)
    print(" ".join(str(t) for t in ids[:a.max_new]))
    print(f"[stats] {len(ids)} tokens, {rate:.1f} tokens/s", file=sys.stderr)
    s.close()


def _trace(a):
    from .trace import replay
    replay(a.model, a.dtype, a.max_tokens, a.out, sys.stdin, lambda text: print(text, flush=True))


def main(argv=None):
    ap = argparse.ArgumentParser(prog="buddy_mlir_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="greedy generation from token ids")
    g.add_argument("--tokens", required=True, help="prompt token ids, separated by commas or blanks")
    g.add_argument("--max-new", type=int, default=32)
    g.add_argument("--max-len", type=int, default=4096, help="positions of the cache")
    g.add_argument("--stop", default="", help="token ids that end the generation")
    g.set_defaults(run=_generate)
    t = sub.add_parser("trace", help="replay steps of token ids and write logits")
    t.add_argument("--out", required=True, help="folder for <step>.f32")
    t.add_argument("--max-tokens", type=int, required=True, help="most tokens live requests hold at any time")
    t.set_defaults(run=_trace)
    for p in (g, t):
        p.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
        p.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    a = ap.parse_args(argv)
    from . import _lib
    _lib.build_if_missing()
    a.run(a)


if __name__ == "__main__":
    main()
