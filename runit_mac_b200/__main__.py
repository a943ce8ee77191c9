"""Command line: ``python -m runit_mac_b200 generate`` (token ids in, token ids out) and ``... trace`` (see trace.py)."""
from __future__ import annotations

import argparse
import sys


def _generate(a) -> int:
    from . import _lib, build
    _lib.load(build.ensure("layered"))
    from . import dispatch, models
    prompt = [int(t) for t in a.tokens.replace(",", " ").split()]
    ctx = dispatch.Context(a.device)
    model = models.load_model(ctx, a.model, a.dtype, max_seq=len(prompt) + a.n + 1)
    if a.temperature > 0:
        cfg = dispatch.SamplerCfg(a.temperature, a.top_k, a.top_p, a.repetition_penalty, 0)
        out = model.generate_sampled(prompt, a.n - 1, cfg, a.seed)[len(prompt) - 1:] if a.n else []
    else:
        out = model.generate(prompt, a.n)
    print(" ".join(str(int(t)) for t in out))
    model.close()
    ctx.close()
    return 0


def _trace(a) -> int:
    from . import trace
    return trace.run(a.model, a.dtype, a.out, a.max_tokens)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="runit_mac_b200")
    sub = ap.add_subparsers(dest="cmd", required=True)
    g = sub.add_parser("generate", help="continue a prompt of token ids")
    g.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    g.add_argument("--tokens", required=True, help="token ids of the prompt, separated by commas or blanks")
    g.add_argument("--n", type=int, default=32, help="tokens to generate")
    g.add_argument("--dtype", default="bfloat16", choices=("bfloat16", "float32"))
    g.add_argument("--temperature", type=float, default=0.0, help="0 = greedy")
    g.add_argument("--top-k", type=int, default=0)
    g.add_argument("--top-p", type=float, default=1.0)
    g.add_argument("--repetition-penalty", type=float, default=1.0)
    g.add_argument("--seed", type=int, default=0)
    g.add_argument("--device", type=int, default=0)
    g.set_defaults(fn=_generate)
    t = sub.add_parser("trace", help="replay token portions from standard input and write logits")
    t.add_argument("--model", required=True)
    t.add_argument("--dtype", default="bfloat16", choices=("bfloat16", "float32"))
    t.add_argument("--out", required=True, help="folder for <step>.f32")
    t.add_argument("--max-tokens", type=int, required=True, help="most tokens a live sequence holds")
    t.set_defaults(fn=_trace)
    a = ap.parse_args(argv)
    return a.fn(a)


if __name__ == "__main__":
    sys.exit(main())
