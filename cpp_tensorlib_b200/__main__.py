"""Command line: ``python -m cpp_tensorlib_b200 generate --model DIR --tokens 1,2,3 -n 16`` (greedy token
ids behind a prompt of ids) and ``... trace --model DIR --out DIR`` (replay of a token trace)."""
import argparse
import sys


def main(argv=None):
    argv = sys.argv[1:] if argv is None else argv
    from . import build
    if argv[:1] == ["trace"]:
        build.build()
        from .trace import main as trace
        return trace(argv[1:])
    ap = argparse.ArgumentParser(prog="cpp_tensorlib_b200", description=__doc__)
    sub = ap.add_subparsers(dest="cmd", required=True)
    g = sub.add_parser("generate", help="greedy generation from token ids")
    g.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    g.add_argument("--tokens", required=True, help="prompt ids, with commas between them")
    g.add_argument("-n", type=int, default=16, help="tokens to generate")
    g.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    g.add_argument("--max-ctx", type=int, default=0, help="capacity in tokens (default: what the call needs)")
    sub.add_parser("trace", help="replay a token trace from standard input")
    a = ap.parse_args(argv)
    build.build()
    from .registry import load_model
    prompt = [int(t) for t in a.tokens.split(",")]
    m = load_model(a.model, a.dtype, a.max_ctx or len(prompt) + a.n)
    print(",".join(map(str, m.generate(prompt, a.n))))
    m.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
