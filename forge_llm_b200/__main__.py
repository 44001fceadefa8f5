"""Command line over a checkpoint folder (config.json, model.safetensors):

    python -m forge_llm_b200 info --model DIR
    python -m forge_llm_b200 generate --model DIR --prompt 3,14,15 [--prompt 9,2,6 ...] [--max-new 32]
        [--dtype bfloat16|float32] [--temperature T --top-k K --top-p P --repeat-penalty R --seed S] [--eos ID,ID]

Prompts are token ids; several prompts run together through the scheduler.  One line of ids per prompt is printed.
"""
from __future__ import annotations

import argparse
import json
import sys


def _ids(text: str) -> list[int]:
    return [int(x) for x in text.replace(",", " ").split()]


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m forge_llm_b200", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    sub = ap.add_subparsers(dest="cmd", required=True)
    p = sub.add_parser("info", help="what a checkpoint holds")
    p.add_argument("--model", required=True)
    g = sub.add_parser("generate", help="continue prompts of token ids")
    g.add_argument("--model", required=True)
    g.add_argument("--prompt", required=True, action="append", type=_ids)
    g.add_argument("--max-new", type=int, default=32)
    g.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    g.add_argument("--device", type=int, default=0)
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--top-k", type=int, default=0)
    g.add_argument("--top-p", type=float, default=0.9)
    g.add_argument("--repeat-penalty", type=float, default=1.1)
    g.add_argument("--seed", type=lambda s: int(s, 0), default=0xDEADBEEF12345678)
    g.add_argument("--eos", type=_ids, default=[])
    g.add_argument("--step-tokens", type=int, default=2048, help="tokens of one scheduler step")
    a = ap.parse_args(argv)
    from .build import ensure_library
    ensure_library()
    from . import engine, runtime
    if a.cmd == "info":
        print(json.dumps(runtime.checkpoint_info(a.model)))
        return 0
    model = runtime.Model.open(a.model, a.dtype, a.device)
    pages = sum(-(-(len(q) + a.max_new) // engine.PAGE) for q in a.prompt)
    eng = engine.Engine(model, pool_tokens=pages * engine.PAGE, slots=len(a.prompt))
    sched = engine.Scheduler(eng, a.step_tokens)
    sampling = engine.Sampling(a.temperature, a.top_k, a.top_p, a.repeat_penalty, a.seed)
    for i, q in enumerate(a.prompt):
        sched.submit(i, q, a.max_new, sampling, a.eos)
    out = sched.run()
    for i in range(len(a.prompt)):
        print(" ".join(map(str, out[i])))
    eng.close()
    model.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
