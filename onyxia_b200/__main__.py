"""Command line: ``python -m onyxia_b200 <command>``.

    models                         the architectures and named configurations this package builds
    generate --model M …           continuous-batching generation from token-id prompts
    trace --model M --out DIR …    replay a trace of batch steps (onyxia_b200/trace.py)

M is a model folder (config.json with model.safetensors) or the name of a built-in configuration with random weights.
"""
from __future__ import annotations

import argparse
import sys


def _ids(text: str) -> list:
    return [int(v) for v in text.replace(",", " ").split()]


def generate(argv) -> int:
    ap = argparse.ArgumentParser(prog="onyxia_b200 generate")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--prompt", action="append", required=True, type=_ids, help="token ids, separated by commas or blanks; repeatable")
    ap.add_argument("-n", "--max-new", type=int, default=32)
    ap.add_argument("--max-tokens", type=int, default=65536, help="cache room over all sequences")
    ap.add_argument("--max-seqs", type=int, default=64)
    ap.add_argument("--token-budget", type=int, default=2048, help="tokens per step")
    ap.add_argument("--eos", type=int, default=-1)
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=0)
    a = ap.parse_args(argv)
    from . import build
    build.ensure_built(oracle=False)
    from . import llm, models
    from .backend import CudaBackend
    from .engine import Engine
    module = models.load_module(a.model, a.dtype)
    if "seq_info" in module.input_names():
        e = Engine(CudaBackend((0,)).prepare(module), a.max_tokens, a.max_seqs)
        outs = e.generate(a.prompt, a.max_new, token_budget=a.token_budget, eos=a.eos, temperature=a.temperature, top_k=a.top_k,
                          top_p=a.top_p, seed=a.seed)
    else:  # a module with dense caches: one sequence after the other
        from .sampling import DeviceSampler, SamplingConfig
        s = llm.NativeLlmSession(CudaBackend((0,)), module, a.max_tokens)
        outs = []
        for p in a.prompt:
            s.reset()
            if a.temperature < 1e-6:
                toks = s.generate(p, a.max_new)
            else:
                sampler = DeviceSampler(s, SamplingConfig(temperature=a.temperature, top_k=a.top_k, top_p=a.top_p, seed=a.seed))
                toks = [sampler.step(p)]
                while len(toks) < a.max_new and toks[-1] != a.eos:
                    toks.append(sampler.step([toks[-1]]))
            outs.append(toks[:toks.index(a.eos) + 1] if a.eos in toks else toks)
    for t in outs:
        print(" ".join(map(str, t)))
    return 0


def main(argv=None) -> int:
    argv = list(sys.argv[1:] if argv is None else argv)
    if argv and argv[0] == "generate":
        return generate(argv[1:])
    if argv and argv[0] == "trace":
        from . import trace
        return trace.main(argv[1:])
    if argv and argv[0] == "models":
        from . import models
        for name in sorted(models.ARCHITECTURES):
            print(f"{name}  (model folders)")
        for name in sorted(models.CONFIGS):
            print(f"{name}  (built-in configuration)")
        return 0
    print(__doc__, file=sys.stderr)
    return 2


if __name__ == "__main__":
    sys.exit(main())
