"""Command line: python -m mllm_b200 {info,generate,trace} --model FOLDER ..."""
import argparse
import sys


def parser():
    ap = argparse.ArgumentParser(prog="mllm_b200", description="Language models on B200.")
    sub = ap.add_subparsers(dest="command", required=True)
    info = sub.add_parser("info", help="what a model folder holds")
    info.add_argument("--model", required=True)
    gen = sub.add_parser("generate", help="greedy continuation of token ids")
    gen.add_argument("--model", required=True)
    gen.add_argument("--tokens", action="append", required=True, help="prompt as comma-separated token ids; repeat for a batch")
    gen.add_argument("--max-new", type=int, default=32)
    gen.add_argument("--stop", default="", help="comma-separated token ids that end a sequence")
    gen.add_argument("--dtype", default=None, help="number format (default: the design's own)")
    gen.add_argument("--slots", type=int, default=8, help="sequences held at once")
    gen.add_argument("--portion", type=int, default=None, help="most prompt tokens of one sequence in a step")
    tr = sub.add_parser("trace", help="replay steps of given tokens from standard input and write logits")
    add_trace_arguments(tr)
    return ap


def add_trace_arguments(ap):
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")


def ids(text):
    return [int(x) for x in text.split(",") if x.strip()]


def trace(args):
    from . import registry, replay
    n = max(args.max_tokens, 1)
    model, runtime = registry.load(args.model, args.dtype, max_seqs=4, max_ctx=n, max_rows=min(n, 4096))
    if runtime != "engine":
        raise SystemExit("only models of the language-model engine replay traces")
    replay.run(model, sys.stdin, args.out, lambda line: print(line, flush=True))
    model.check_device_status()
    model.close()


def main(argv=None):
    args = parser().parse_args(argv)
    from . import registry
    if args.command == "info":
        cfg = registry.read_config(args.model)
        name = registry.architecture(cfg)
        runtime, dtypes, _ = registry.MODELS[name]
        print(f"{name}: runtime {runtime}, number formats {', '.join(dtypes)}")
    elif args.command == "generate":
        prompts = [ids(t) for t in args.tokens]
        ctx = max(len(p) for p in prompts) + args.max_new
        model, runtime = registry.load(args.model, args.dtype, max_seqs=min(args.slots, len(prompts)), max_ctx=ctx,
                                       max_rows=min(4096, sum(len(p) for p in prompts)))
        for out in registry.generate(model, runtime, prompts, args.max_new, set(ids(args.stop)), args.portion):
            print(",".join(str(t) for t in out))
        model.close()
    else:
        trace(args)


if __name__ == "__main__":
    main()
