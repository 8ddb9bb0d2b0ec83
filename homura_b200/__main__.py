"""Command line over token ids.

    python -m homura_b200 info MODEL                 config and tensors of a checkpoint (no GPU needed)
    python -m homura_b200 generate MODEL --ids 1,2,3 [--ids 4,5 ...] [--max-new 32] [--temperature T ...]

MODEL is a folder with config.json and safetensors (any design the library knows) or a .gguf file.  generate runs all
prompts through one continuous-batching scheduler and prints one line of ids per prompt; it is greedy unless a
temperature is given.
"""
from __future__ import annotations

import argparse
import sys

from . import DType, HfModel, SamplingConfig, checkpoint_info


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m homura_b200", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    sub = ap.add_subparsers(dest="command", required=True)
    p = sub.add_parser("info")
    p.add_argument("model")
    p = sub.add_parser("generate")
    p.add_argument("model")
    p.add_argument("--ids", action="append", required=True, help="token ids of one prompt, separated by commas; may be given several times")
    p.add_argument("--max-new", type=int, default=32)
    p.add_argument("--dtype", choices=["bf16", "f32"], default="bf16", help="f32: f32 cache pages, and f32 projections where the design has them")
    p.add_argument("--slots", type=int, default=8, help="requests that run at once")
    p.add_argument("--pool-tokens", type=int, default=0, help="cache size in tokens (default: enough for --slots of the longest prompt)")
    p.add_argument("--temperature", type=float, default=0.0)
    p.add_argument("--top-k", type=int, default=50)
    p.add_argument("--top-p", type=float, default=0.9)
    p.add_argument("--repetition-penalty", type=float, default=1.0)
    p.add_argument("--seed", type=int, default=0)
    args = ap.parse_args(argv)

    if args.command == "info":
        info = checkpoint_info(args.model)
        for k, v in info["config"].items():
            if k != "layers":
                print(f"{k}: {v}")
        for i, layer in enumerate(info["config"].get("layers", [])):
            print(f"layer {i}: {layer}")
        for t in info["tensors"]:
            print(f"{t['name']}  {t['dtype']}  {t['shape']}")
        return 0

    from .serving import Scheduler, Session

    prompts = [[int(t) for t in s.split(",")] for s in args.ids]
    dtype = DType.BF16 if args.dtype == "bf16" else DType.F32
    model = HfModel.load_gguf(args.model) if args.model.endswith(".gguf") else HfModel.load_with_dtype(args.model, dtype)
    need = max(map(len, prompts)) + args.max_new
    slots = max(1, min(args.slots, len(prompts)))
    session = Session(model, slots, args.pool_tokens or slots * (need + 64), kv_dtype=dtype, max_seq_len=need + 64)
    sampling = None
    if args.temperature > 0 or args.repetition_penalty != 1.0:
        sampling = SamplingConfig(temperature=args.temperature, top_k=args.top_k, top_p=args.top_p, repetition_penalty=args.repetition_penalty, seed=args.seed)
    for ids in Scheduler(session).run(prompts, args.max_new, sampling):
        print(",".join(map(str, ids)))
    return 0


if __name__ == "__main__":
    sys.exit(main())
