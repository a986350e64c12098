"""Command line.

    python -m lithos_b200 generate --model DIR --prompt-ids 1,2,3 [--max-new N] [--eos ID] [--temperature T --top-k K --seed S]
    python -m lithos_b200 architectures

Token ids in, token ids out (no tokenizer).  The model class is chosen by DIR/config.json."""
import argparse
import json
import sys
import time


def main(argv=None):
    ap = argparse.ArgumentParser(prog="lithos_b200")
    sub = ap.add_subparsers(dest="cmd", required=True)
    g = sub.add_parser("generate", help="prompt pass, then tokens until EOS or the limit")
    g.add_argument("--model", required=True)
    g.add_argument("--prompt-ids", required=True, help="comma-separated token ids")
    g.add_argument("--max-new", type=int, default=32)
    g.add_argument("--max-ctx", type=int, default=None, help="positions the caches hold (default: prompt + new tokens)")
    g.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    g.add_argument("--eos", type=int, default=-1)
    g.add_argument("--temperature", type=float, default=1.0)
    g.add_argument("--top-k", type=int, default=0, help="0: greedy")
    g.add_argument("--seed", type=int, default=0)
    g.add_argument("--device", type=int, default=0)
    sub.add_parser("architectures", help="model classes of the registry")
    a = ap.parse_args(argv)
    if a.cmd == "architectures":
        from . import build, model
        build(images=[])
        print("\n".join(model.architectures()))
        return 0
    from .serve import open_model
    prompt = [int(t) for t in a.prompt_ids.split(",")]
    ctx, m = open_model(a.model, a.max_ctx or len(prompt) + a.max_new, a.dtype, a.device)
    if a.top_k:
        m.set_sampling(a.temperature, a.top_k, a.seed)
    t0 = time.perf_counter()
    out = m.generate(prompt, a.max_new, a.eos)
    print(json.dumps({"tokens": out, "seconds": round(time.perf_counter() - t0, 4)}))
    m.close()
    ctx.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
