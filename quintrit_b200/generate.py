"""Generation from the command line.

    python -m quintrit_b200.generate --model PATH --prompt TEXT | --tokens 1,2,3  [--max-new N] [--temperature T --top-k K --top-p P --seed S]

PATH is a GGUF file or a model folder. Text goes through the model's tokenizer and is streamed; ``--tokens`` takes and prints token ids,
for models without one. Temperature 0 (the default) is greedy.
"""
from __future__ import annotations

import argparse
import sys

from .api import QuintritError
from .runtime import Model


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m quintrit_b200.generate", description="Generates text or token ids with a model on a B200.")
    ap.add_argument("--model", required=True, help="GGUF file or model folder (config.json + model.safetensors)")
    src = ap.add_mutually_exclusive_group(required=True)
    src.add_argument("--prompt", help="text")
    src.add_argument("--tokens", help="token ids, with commas between them; ids are printed the same way")
    ap.add_argument("--max-new", type=int, default=64)
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--top-k", type=int, default=40)
    ap.add_argument("--top-p", type=float, default=0.9)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--device", default="cuda")
    ap.add_argument("--context", type=int, default=None)
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default=None, help="arithmetic of a model folder")
    a = ap.parse_args(argv)
    try:
        model = Model.load(a.model, device=a.device, context=a.context, dtype=a.dtype)
        kw = dict(temperature=a.temperature, top_k=a.top_k, top_p=a.top_p, seed=a.seed)
        if a.tokens is not None:
            print(",".join(str(t) for t in model.new_session().sample_tokens([int(t) for t in a.tokens.split(",")], a.max_new, **kw)))
        else:
            for piece in model.stream(a.prompt, a.max_new, **kw):
                print(piece, end="", flush=True)
            print()
    except QuintritError as e:
        print(f"error: {e}", file=sys.stderr)
        return 1
    return 0


if __name__ == "__main__":
    sys.exit(main())
