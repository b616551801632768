"""Command line: continue prompts of token ids with any model of the registry, several at a time (slot scheduler).

    python -m seq2seqsharp_b200.cli generate --model DIR [--max-new 32] [--slots 4] [--top-p 0.9 --temperature 1.0 --seed 1] < prompts
    python -m seq2seqsharp_b200.cli info --model DIR

One prompt per line of standard input (ids separated by blanks); one line of generated ids per prompt on standard output, in order.
Generation of a prompt ends with id 0 (</s>), which is printed, or after --max-new tokens.
"""
import argparse
import sys

from .gpt import DecodingOptions, DecodingStrategyEnums


def _options(a, max_tokens):
    sampling = a.top_p < 1.0 or a.temperature != 1.0
    return DecodingOptions(MaxTgtSentLength=max_tokens, TopP=a.top_p, Temperature=a.temperature, RepeatPenalty=a.repeat_penalty, Seed=a.seed,
                           DecodingStrategy=DecodingStrategyEnums.Sampling if sampling else DecodingStrategyEnums.GreedySearch,
                           BlockedTokens=[0] if a.ignore_eos else None)


def generate(gpt, prompts, opts, slots: int, max_new: int):
    """Generated ids per prompt through the slot scheduler."""
    from .scheduler import ContinuousBatcher, Request
    out = ContinuousBatcher(gpt, opts, slots=slots, max_tokens=gpt.max_tokens).run([Request(i, p, max_new) for i, p in enumerate(prompts)])
    return [[int(t) for t in out[i]] for i in range(len(prompts))]


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="seq2seqsharp_b200.cli")
    sub = ap.add_subparsers(dest="cmd", required=True)
    g = sub.add_parser("generate", help="continue prompts of token ids read from standard input")
    i = sub.add_parser("info", help="what a model folder holds (needs no GPU)")
    for p in (g, i):
        p.add_argument("--model", required=True, help="model folder (config.json, model.safetensors) or a reference model file")
        p.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    g.add_argument("--device", type=int, default=0)
    g.add_argument("--max-new", type=int, default=32)
    g.add_argument("--slots", type=int, default=4, help="sequences in flight")
    g.add_argument("--top-p", type=float, default=1.0)
    g.add_argument("--temperature", type=float, default=1.0)
    g.add_argument("--repeat-penalty", type=float, default=2.0)
    g.add_argument("--seed", type=int, default=0)
    g.add_argument("--ignore-eos", action="store_true", help="never choose id 0")
    a = ap.parse_args(argv)
    from . import registry
    if a.cmd == "info":
        _, cfg = registry.read_config(a.model, a.dtype)
        n = sum(int(r) * int(c) for r, c in cfg.weight_shapes().values())
        print("%s: %d layers, width %d, vocabulary %d, %d values in %d tensors, %d multiply-adds per token" %
              (cfg.name, cfg.L, cfg.d, cfg.V, n, len(cfg.weight_shapes()), cfg.active_matmul_params()))
        return 0
    prompts = [[int(t) for t in line.split()] for line in sys.stdin if line.strip()]
    if not prompts:
        return 0
    max_tokens = max(len(p) for p in prompts) + a.max_new + 2
    slots = max(1, min(a.slots, len(prompts)))
    gpt = registry.load_model(a.model, dtype=a.dtype, device_id=a.device, max_batch=slots, max_tokens=max_tokens)
    for ids in generate(gpt, prompts, _options(a, max_tokens), slots, a.max_new):
        print(" ".join(map(str, ids)))
    gpt.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
