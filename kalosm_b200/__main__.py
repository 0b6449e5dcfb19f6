"""Command line: generate token ids with any registered model.

  python -m kalosm_b200 --model PATH --tokens 5,17,3 --steps 32 [--sample --temperature 0.8 --top-k 64 --seed 1]

PATH is a checkpoint folder (config.json, model.safetensors) or a GGUF file. Greedy unless --sample is given.
"""
import argparse
import json
import sys


def main(argv=None):
    ap = argparse.ArgumentParser(prog="python -m kalosm_b200", description="generate token ids with a checkpoint")
    ap.add_argument("--model", required=True, help="checkpoint folder or GGUF file")
    ap.add_argument("--tokens", required=True, help="prompt as token ids with commas between them")
    ap.add_argument("--steps", type=int, default=32)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--max-seq-len", type=int, default=0)
    ap.add_argument("--sample", action="store_true", help="sample instead of the greedy token")
    ap.add_argument("--temperature", type=float, default=0.8)
    ap.add_argument("--top-k", type=int, default=64)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=0)
    args = ap.parse_args(argv)
    import kalosm_b200 as kb
    from . import models
    prompt = [int(t) for t in args.tokens.split(",")]
    model = models.load_model(kb.Device(0), args.model, max_seq_len=args.max_seq_len or len(prompt) + args.steps + 1, dtype=args.dtype)
    out = generate(model, prompt, args.steps, kb.SamplerConfig(temperature=args.temperature, top_k=args.top_k, top_p=args.top_p,
                                                               seed=args.seed) if args.sample else None)
    print(json.dumps({"prompt": prompt, "generated": out}))
    return 0


def generate(model, prompt, steps, sampler=None):
    """Prompt pass up to the last prompt token, then the device-resident loop from that token on."""
    model.reset()
    if len(prompt) > 1:
        model.forward(prompt[:-1], want_logits=False)
    last = [prompt[-1]]
    ids = model.generate_sampled(last, steps, sampler) if sampler is not None else model.generate_greedy(last, steps)
    return [int(t) for t in ids[0]]


if __name__ == "__main__":
    sys.exit(main())
