"""Command line: `python -m hologram_b200 generate --model DIR --tokens 1,2,3 --max-new 16`."""
import argparse
import sys


def main(argv=None):
    ap = argparse.ArgumentParser(prog="hologram_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="continue token prompts with a model")
    g.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    g.add_argument("--tokens", required=True, action="append", help="a prompt: token ids with commas between them (repeat for more prompts)")
    g.add_argument("--max-new", type=int, default=16)
    g.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--top-k", type=int, default=0)
    g.add_argument("--seed", type=int, default=0)
    g.add_argument("--portion", type=int, default=0, help="most prompt tokens per step (0 = the runner's largest)")
    g.add_argument("--device", type=int, default=0)
    sub.add_parser("models", help="list the architectures that can be loaded")
    a = ap.parse_args(argv)
    from . import models
    if a.command == "models":
        print("\n".join(sorted(models.ARCHITECTURES)))
        return 0
    from . import decode
    from .backend import B200Backend
    prompts = [[int(t) for t in p.split(",")] for p in a.tokens]
    model = models.load_model(a.model, a.dtype)
    backend = B200Backend(a.device)
    runner = decode.StepRunner(backend, model, max(len(p) for p in prompts) + a.max_new)
    scheduler = decode.Scheduler(runner, a.portion or None)
    requests = [decode.Request(p, a.max_new, decode.Sampler(a.temperature, a.top_k, a.seed + i)) for i, p in enumerate(prompts)]
    for r in requests:
        scheduler.submit(r)
    for _ in scheduler.run():
        pass
    for r in requests:
        print(",".join(str(t) for t in r.tokens))
    runner.close()
    backend.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
