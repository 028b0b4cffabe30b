"""Command line: `python -m det_b200 generate --model PATH --prompt 1,2,3 --new 16` continues token ids with any registered
checkpoint (a model folder or a det GGUF); `python -m det_b200 models` lists the architectures.  Token ids in, token ids out:
there is no tokenizer here."""
from __future__ import annotations

import argparse
import ctypes as C
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="det_b200")
    sub = ap.add_subparsers(dest="cmd", required=True)
    g = sub.add_parser("generate", help="prefill token ids and generate")
    g.add_argument("--model", required=True, help="model folder or det GGUF file")
    g.add_argument("--prompt", required=True, help="token ids, comma separated")
    g.add_argument("--new", type=int, default=16, help="tokens to generate")
    g.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    g.add_argument("--temperature", type=float, default=0.0, help="0: greedy")
    g.add_argument("--top-k", type=int, default=0)
    g.add_argument("--top-p", type=float, default=1.0)
    g.add_argument("--seed", type=int, default=0)
    g.add_argument("--max-batch", type=int, default=512, help="tokens per prefill step")
    sub.add_parser("models", help="list the registered architectures")
    a = ap.parse_args(argv)
    from . import build, capi
    build.build_all()
    if a.cmd == "models":
        buf = C.create_string_buffer(4096)
        capi.host().dh_architectures(buf, len(buf))
        print("\n".join(buf.value.decode().split()))
        return 0
    from .engine import Engine, EngineError
    prompt = [int(t) for t in a.prompt.split(",") if t.strip()]
    try:
        e = Engine.open(a.model, a.dtype, max_ctx=len(prompt) + a.new, max_batch=min(a.max_batch, len(prompt) + a.new))
        print(",".join(str(t) for t in e.generate(prompt, a.new, a.temperature, a.top_k, a.top_p, a.seed)))
        e.close()
    except EngineError as ex:
        print(f"det_b200: {ex}", file=sys.stderr)
        return 1
    return 0


if __name__ == "__main__":
    sys.exit(main())
