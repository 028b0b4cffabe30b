"""Replays a trace: given token ids go through a model step by step, and chosen logits are written to files.

Steps come from standard input, one JSON object a line:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
An entry carries a request's next tokens and the places among them whose logits are wanted; `end` names requests that are
over after the step.  A step with wanted logits writes OUT/<step>.f32 (little-endian fp32, [wanted, vocab], in the order of
the entries and of `want`); every step is answered by a line `done <step>`.
"""
from __future__ import annotations

import argparse
import json
import os
import sys



class Replayer:
    """Keeps a sequence (caches and states) per live request; ended requests give theirs to later ones."""

    def __init__(self, engine, max_tokens: int):
        self.engine, self.max_tokens = engine, max_tokens
        self.live: dict[str, int] = {}
        self.free: list[int] = []

    def entry(self, rid: str, tokens, want):
        if rid not in self.live:
            self.live[rid] = self.free.pop() if self.free else self.engine.new_sequence(self.max_tokens)
        seq = self.live[rid]
        self.engine.swap(seq)
        try:
            return self.engine.step(tokens, want)
        finally:
            self.engine.swap(seq)

    def end(self, rid: str) -> None:
        seq = self.live.pop(rid, None)
        if seq is not None:
            self.engine.clear(seq)
            self.free.append(seq)

    def close(self) -> None:
        for seq in list(self.live.values()) + self.free:
            self.engine.free(seq)
        self.live, self.free = {}, []


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay given tokens through a model and write chosen logits.")
    ap.add_argument("--model", required=True, help="model folder (config.json, model.safetensors) or det GGUF file")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits files")
    ap.add_argument("--max-tokens", type=int, required=True, help="the most tokens live requests hold at any time")
    a = ap.parse_args(argv)

    from . import build
    build.build_all()
    from .engine import Engine
    max_tokens = max(1, a.max_tokens)
    engine = Engine.open(a.model, a.dtype, max_ctx=max_tokens, max_batch=min(max_tokens, 1024))
    replay = Replayer(engine, max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = [replay.entry(e["id"], e["tokens"], e.get("want", [])) for e in step["entries"]]
        if any(len(r) for r in rows):
            path = os.path.join(a.out, f"{step['step']}.f32")
            with open(path, "wb") as f:
                for r in rows:
                    if sys.byteorder != "little":
                        r.byteswap()
                    f.write(r.tobytes())
        for rid in step.get("end", []):
            replay.end(rid)
        print(f"done {step['step']}", flush=True)
    replay.close()
    engine.close()
    return 0
