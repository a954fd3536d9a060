"""Generates from token ids with any model the registry knows.

    python -m camelid_b200.generate --model PATH --tokens 1,2,3 [--tokens 4,5] -n 32 [--temperature T --min-p P --seed S]

Several --tokens are decoded together.  Prints one line of generated ids per prompt."""
from __future__ import annotations

import argparse


def main(argv=None):
    ap = argparse.ArgumentParser(prog="camelid_b200.generate", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="a GGUF file, or a folder with config.json and model.safetensors")
    ap.add_argument("--tokens", action="append", required=True, help="prompt as comma-separated token ids; may be repeated")
    ap.add_argument("-n", "--max-new", type=int, default=32)
    ap.add_argument("--dtype", default=None, help="bfloat16 (default) or float32, for models that offer the choice")
    ap.add_argument("--max-pos", type=int, default=0, help="context length (default: what the prompts need)")
    ap.add_argument("--portion", type=int, default=0, help="feed prompts in portions of this many tokens")
    ap.add_argument("--temperature", type=float, default=0.0, help="0 = greedy")
    ap.add_argument("--min-p", type=float, default=0.0)
    ap.add_argument("--seed", type=int, default=0)
    a = ap.parse_args(argv)
    from . import models
    from .scheduler import Scheduler

    prompts = [[int(t) for t in p.split(",")] for p in a.tokens]
    max_pos = a.max_pos or max(len(p) for p in prompts) + a.max_new
    eng = models.load_model(a.model, max_pos=max_pos, max_seqs=len(prompts), dtype=a.dtype)
    s = Scheduler(eng, portion=a.portion)
    for i, p in enumerate(prompts):
        s.submit(i, p, a.max_new, a.temperature, a.min_p, a.seed + 1000003 * i)
    out = s.run()
    for i in range(len(prompts)):
        print(",".join(str(t) for t in out[i]), flush=True)
    eng.close()


if __name__ == "__main__":
    main()
