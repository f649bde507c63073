"""Replays a trace of token ids through a model, step by step, and writes the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps

Standard input has one JSON object per line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["a"]}

An entry brings the next tokens of a request and the places among them whose logits are wanted; ``end`` lists the requests that
are over.  For a step with wanted places OUT/<step>.f32 holds them as little-endian f32 [wanted, vocab]; after every step a line
``done <step>`` is printed.  The tokens go through the session that generation uses, which holds one request at a time: a step of a new
request is refused until the previous one has ended.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

DTYPES = {"bfloat16": "bf16", "float32": "f32"}
PREFILL = 512  # longest prefill chunk of a replay


def replay(session, vocab: int, lines, out_dir: str, emit) -> None:
    """Run the steps in ``lines`` on an LlmSession; ``emit`` receives every line to print."""
    current = None
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        blocks = []
        for e in step.get("entries", ()):
            if e["id"] != current:
                if current is not None:
                    raise ValueError(f"request {e['id']!r} begins before {current!r} has ended")
                session.reset()
                current = e["id"]
            want = e.get("want") or []
            logits = session.feed(e["tokens"], want)
            if want:
                blocks.append(logits.numpy().astype("<f4", copy=False).tobytes())
        if blocks:
            with open(os.path.join(out_dir, f"{step['step']}.f32"), "wb") as f:
                f.write(b"".join(blocks))
        if current in (step.get("end") or ()):
            session.reset()
            current = None
        emit(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay token ids through a model and write logits.")
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=sorted(DTYPES))
    ap.add_argument("--out", required=True, help="directory for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that a request holds")
    args = ap.parse_args(argv)
    from . import build
    build.build()  # compiles what is missing or older than its sources
    from .registry import load_model
    from .session import LlmSession
    length = max(args.max_tokens, 1)
    model = load_model(args.model, dtype=DTYPES[args.dtype], max_seq_len=length, output="logits", max_prefill=min(PREFILL, length))
    session = LlmSession.for_model(model, eos_token_id=-1, prefill_len=model.max_prefill)

    def emit(text):
        sys.stdout.write(text + "\n")
        sys.stdout.flush()

    replay(session, model.vocab, iter(sys.stdin.readline, ""), args.out, emit)
    model.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
