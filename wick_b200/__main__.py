"""Command line over token ids (there is no tokenizer here):

    python -m wick_b200 info     --model PATH
    python -m wick_b200 generate --model PATH --tokens 1,2,3 [--count N] [--temperature T --top-k K --top-p P --seed S]
    python -m wick_b200 trace    --model PATH --out DIR < steps        (the same as bin/trace_run)

PATH is a GGUF file or a folder with config.json and model.safetensors; the model class is chosen by what it holds.
"""
from __future__ import annotations

import argparse
import sys

import numpy as np


def _load(args):
    from . import build
    build.build()
    from .model import load_model_cuda
    return load_model_cuda(args.model, args.context, args.device, args.dtype)


def _info(args) -> int:
    m = _load(args)
    c = m.config()
    print(f"architecture {c.architecture}: {c.n_layers} layers, width {c.hidden_size}, vocabulary {c.vocab_size}, {m.gpu_memory_bytes() / 1e6:.0f} MB on the device")
    for i, t in enumerate(c.block_types):
        print(f"  layer {i}: {t}" + (f", {c.kv_heads_per_layer[i]} key/value heads" if c.kv_heads_per_layer[i] else ""))
    return 0


def _generate(args) -> int:
    from .model import InferenceState
    m = _load(args)
    st = InferenceState()
    prompt = [int(t) for t in args.tokens.replace(",", " ").split()]
    _, logits = m.forward_prefill_chunked(prompt, 0, st, args.ubatch)
    rng = np.random.default_rng(args.seed)
    out = [int(np.argmax(logits))] if args.temperature <= 0 else []
    if args.temperature <= 0:
        out += [int(t) for t in m.generate_greedy(out[0], args.count - 1, st)] if args.count > 1 else []
    else:
        # the sampler runs on the logits of a decode step: the last prompt token is fed again as that step
        m.forward_prefill_chunked(prompt[:-1], 0, st, args.ubatch) if len(prompt) > 1 else m.reset(st)
        tok = prompt[-1]
        for i in range(args.count):
            tok = m.forward_sample([tok], len(prompt) - 1 + i, st, args.temperature, args.top_k, args.top_p, float(rng.random(dtype=np.float32)))
            out.append(tok)
    print(*out[:args.count])
    return 0


def main(argv=None) -> int:
    argv = sys.argv[1:] if argv is None else argv
    if argv and argv[0] == "trace":
        from . import trace
        return trace.main(argv[1:])
    ap = argparse.ArgumentParser(prog="wick_b200", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    sub = ap.add_subparsers(dest="command", required=True)
    for name, fn in (("info", _info), ("generate", _generate)):
        p = sub.add_parser(name)
        p.set_defaults(fn=fn)
        p.add_argument("--model", required=True)
        p.add_argument("--context", type=int, default=4096)
        p.add_argument("--device", type=int, default=0)
        p.add_argument("--dtype", default="default", choices=["default", "bfloat16", "float32"])
        if name == "generate":
            p.add_argument("--tokens", required=True, help="prompt token ids, separated by commas or spaces")
            p.add_argument("--count", type=int, default=16)
            p.add_argument("--ubatch", type=int, default=512)
            p.add_argument("--temperature", type=float, default=0.0)
            p.add_argument("--top-k", type=int, default=40)
            p.add_argument("--top-p", type=float, default=1.0)
            p.add_argument("--seed", type=int, default=0)
    args = ap.parse_args(argv)
    return args.fn(args)


if __name__ == "__main__":
    sys.exit(main())
