"""Greedy generation from a model folder: `python -m popxl_addons_b200.generate --model DIR --prompt "5 17 3" --prompt "8"`.
Prompts are token ids; one line of token ids is printed per prompt."""
import argparse
import sys

__all__ = ["main"]


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="popxl_addons_b200.generate", description="Greedy generation from token ids.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--prompt", action="append", required=True, help="token ids separated by spaces or commas; repeatable")
    ap.add_argument("--max-new-tokens", type=int, default=32)
    ap.add_argument("--dtype", default="bfloat16", choices=("bfloat16", "float32"))
    ap.add_argument("--batch", type=int, default=0, help="sequences run together (default: all prompts, at most 16)")
    ap.add_argument("--max-seq", type=int, default=0, help="positions a sequence can hold (default: what the prompts need)")
    ap.add_argument("--device", default="auto")
    a = ap.parse_args(argv)
    from .models.registry import load_model

    prompts = [[int(x) for x in p.replace(",", " ").split()] for p in a.prompt]
    need = max(len(p) for p in prompts) + a.max_new_tokens
    gen = load_model(a.model, dtype=a.dtype, batch=a.batch or min(len(prompts), 16), max_seq=a.max_seq or need,
                     max_new_tokens=a.max_new_tokens, device=a.device)
    for out in gen.generate(prompts, a.max_new_tokens):
        print(" ".join(str(int(x)) for x in out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
