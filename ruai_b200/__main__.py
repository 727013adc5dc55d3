"""Command line: `python -m ruai_b200 generate --model DIR --ids 1,2,3 -n 16`, `python -m ruai_b200 info --model DIR`.

There is no tokenizer here: prompts and results are token ids.
"""
import argparse
import sys

from . import nn, registry


def main(argv=None):
    ap = argparse.ArgumentParser(prog="ruai_b200")
    sub = ap.add_subparsers(dest="cmd", required=True)
    g = sub.add_parser("generate", help="continue a prompt of token ids")
    g.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    g.add_argument("--ids", required=True, help="the prompt: token ids with commas between them")
    g.add_argument("-n", type=int, default=16, help="tokens to generate")
    g.add_argument("--dtype", default="bfloat16", choices=registry.DTYPES, help="number format of models that run unquantized")
    g.add_argument("--bits", type=int, choices=(4, 8), help="quantize an unquantized Llama / GPT-2 checkpoint")
    g.add_argument("--group", type=int, default=32)
    g.add_argument("--temperature", type=float, default=0.0, help="0: greedy")
    g.add_argument("--top-k", type=int, default=0)
    g.add_argument("--top-p", type=float, default=1.0)
    g.add_argument("--seed", type=int, default=0)
    i = sub.add_parser("info", help="which model of the registry serves a folder")
    i.add_argument("--model", required=True)
    a = ap.parse_args(argv)
    if a.cmd == "info":
        print(registry.architecture(registry.read_config(a.model)))
        return 0
    m = registry.load(nn.Device.cuda(0), a.model, a.dtype, a.bits, a.group)
    ids = [int(x) for x in a.ids.split(",")]
    out = m.generate_sampled(ids, a.n, a.temperature, a.top_k, a.top_p, a.seed) if a.temperature > 0 else m.generate(ids, a.n)
    print(",".join(str(int(x)) for x in out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
