"""Greedy generation from the command line, for every model family of the registry.

    python -m my_nn_engine_b200.generate --model DIR --prompt-ids 1,2,3 [--max-new-tokens 16] [--dtype bf16] [--max-seq-len 2048]
                                         [--prefill 512] [--eos ID] [--tokenizer tokenizer.json --prompt TEXT]

Prints the new token ids (or the text, with a tokenizer).
"""
from __future__ import annotations

import argparse
import sys

from .registry import load_model, read_config
from .session import LlmSession


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m my_nn_engine_b200.generate", description="Greedy generation from a model directory.")
    ap.add_argument("--model", required=True, help="directory with config.json and safetensors weights")
    ap.add_argument("--prompt-ids", help="comma-separated token ids")
    ap.add_argument("--prompt", help="text prompt (needs --tokenizer)")
    ap.add_argument("--tokenizer", help="tokenizer.json")
    ap.add_argument("--max-new-tokens", type=int, default=16)
    ap.add_argument("--dtype", default="bf16", choices=["bf16", "f16", "f32"])
    ap.add_argument("--max-seq-len", type=int, default=2048)
    ap.add_argument("--prefill", type=int, default=512, help="longest prefill chunk")
    ap.add_argument("--eos", type=int, help="end-of-sequence id (default: the configuration's, if it has one)")
    args = ap.parse_args(argv)
    if (args.prompt_ids is None) == (args.prompt is None):
        ap.error("give either --prompt-ids or --prompt")
    tok = None
    if args.tokenizer:
        from tokenizers import Tokenizer
        tok = Tokenizer.from_file(args.tokenizer)
    eos = args.eos
    if eos is None:
        eos = read_config(args.model).get("eos_token_id")
        eos = eos[0] if isinstance(eos, list) else eos
    model = load_model(args.model, dtype=args.dtype, max_seq_len=args.max_seq_len, output="ids", max_prefill=args.prefill)
    # the session counts a prompt in whole prefill chunks; keep them from exceeding the cache
    session = LlmSession.for_model(model, -1 if eos is None else eos, prefill_len=min(args.prefill, args.max_seq_len), tokenizer=tok)
    prompt = args.prompt if args.prompt is not None else [int(t) for t in args.prompt_ids.split(",") if t.strip()]
    ids = session.generate_ids(prompt, args.max_new_tokens)
    print(tok.decode(ids) if tok else ",".join(str(t) for t in ids))
    model.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
