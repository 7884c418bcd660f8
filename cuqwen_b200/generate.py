"""Greedy generation from the command line, for every kind of model the library opens.

    python -m cuqwen_b200.generate --model DIR --tokens 5,17,3 -n 32                       # a model directory (config.json + model.safetensors)
    python -m cuqwen_b200.generate --model FILE.bin --size 7b --quant int4 --ranks RANKS.json --prompt "Hello" -n 64   # a weight file of the table's models

The prompt goes through the batched prefill, the rest through the decode step; the generated ids (and, with --ranks, the
text) are printed.
"""
from __future__ import annotations

import argparse
import sys
from pathlib import Path

from . import engine as E


def open_engine(a) -> E.Engine:
    if Path(a.model).is_dir():
        return E.Engine.open(a.model, act=a.dtype, max_seq_len=a.max_seq_len, device=a.device, repetition_penalty=a.repetition_penalty)
    if not a.size:
        raise SystemExit("a weight file needs --size and --quant (a model directory names its design itself)")
    p = E.model_params(a.size, a.quant)
    p.device, p.repetition_penalty = a.device, a.repetition_penalty or p.repetition_penalty
    if a.max_seq_len:
        p.max_seq_len = a.max_seq_len
    eng = E.Engine(p)
    eng.load(a.model)
    return eng


def parser() -> argparse.ArgumentParser:
    ap = argparse.ArgumentParser(prog="python -m cuqwen_b200.generate", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="model directory or weight file")
    ap.add_argument("--dtype", default="bfloat16", choices=sorted(E.ACT_ID), help="activations of a model directory's design")
    ap.add_argument("--size", default="", choices=["", *E.MODEL_ID], help="weight file: row of the model table")
    ap.add_argument("--quant", default="int4", choices=sorted(E.QUANT_ID), help="weight file: weight format")
    ap.add_argument("--tokens", default="", help="prompt as token ids, with commas or spaces between them")
    ap.add_argument("--prompt", default="", help="prompt as text (needs --ranks)")
    ap.add_argument("--ranks", default="", help="tokenizer ranks file (export.py writes one)")
    ap.add_argument("-n", type=int, default=32, help="tokens to generate")
    ap.add_argument("--repetition-penalty", type=float, default=0.0, help="penalise ids that have been seen (0: no penalty)")
    ap.add_argument("--max-seq-len", type=int, default=0)
    ap.add_argument("--device", type=int, default=0)
    return ap


def main(argv=None) -> int:
    a = parser().parse_args(argv)
    tok = None
    if a.ranks:
        from .tokenizer import QwenTokenizer
        tok = QwenTokenizer(a.ranks)
    if a.prompt and not tok:
        raise SystemExit("--prompt needs --ranks")
    ids = tok.encode(a.prompt) if a.prompt else [int(t) for t in a.tokens.replace(",", " ").split()]
    if not ids:
        raise SystemExit("the prompt is empty: give --tokens or --prompt")
    eng = open_engine(a)
    out = [int(t) for t in eng.generate(ids, a.n, penalise=a.repetition_penalty > 0)]
    eng.close()
    print(*out)
    if tok:
        print(tok.decode(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
