"""Sampler (the reference's scripts/sample.py:1-7 is a stub): load a checkpoint, encode a prompt
with the GPT-2 BPE, generate with the KV cache, decode and print.

    python scripts/sample.py --checkpoint_dir checkpoints/ --prompt "Hello" --new_tokens 50 --top_k 40
    python scripts/sample.py --preset gpt2-tiny --random-weights --prompt "abc"
    python scripts/sample.py --model-dir DIR --prompt-ids 12,40,7        # any registered family that loads from a folder
"""
from __future__ import annotations

import argparse
import sys

from utils import get_tokenizer, gpt_config

import torch


def main(argv=None):
    from jax_gpt_b200.models.gpt2 import GPT
    ap = argparse.ArgumentParser(description=__doc__)
    ap.add_argument("--preset", default="gpt2")
    ap.add_argument("--checkpoint_dir", default="")
    ap.add_argument("--step", type=int, default=-1, help="-1 = latest")
    ap.add_argument("--hf", default="", help="load HF weights by name or path instead of a checkpoint")
    ap.add_argument("--random-weights", action="store_true")
    ap.add_argument("--prompt", default="Hello, my name is")
    ap.add_argument("--model-dir", default="", help="folder with config.json and *.safetensors; the class is chosen by config.json")
    ap.add_argument("--prompt-ids", action="append", default=[], help="with --model-dir: comma-separated token ids (repeatable)")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"], help="with --model-dir")
    ap.add_argument("--new_tokens", type=int, default=32)
    ap.add_argument("--temperature", type=float, default=1.0)
    ap.add_argument("--top_k", type=int, default=0)
    ap.add_argument("--num_samples", type=int, default=1)
    ap.add_argument("--seed", type=int, default=0)
    args = ap.parse_args(argv)
    if args.model_dir:
        return sample_from_folder(args)

    cfg = gpt_config(args.preset)
    if args.hf:
        model = GPT.from_pretrained(args.hf)
    else:
        model = GPT(cfg, seed=args.seed)
        if args.checkpoint_dir and not args.random_weights:
            from jax_gpt_b200.trainer import TrainConfig, create_optimizer, create_train_state
            from jax_gpt_b200.trainer.checkpointing import CheckpointManager
            tc = TrainConfig(checkpoint_dir=args.checkpoint_dir)
            state = create_train_state(model, create_optimizer(model, tc))
            state = CheckpointManager(tc, cfg).restore(None if args.step < 0 else args.step, state)
            print(f"loaded checkpoint step {state.step}")
    tok = get_tokenizer()
    ids = tok.encode(args.prompt) or [tok.eot]
    idx = torch.tensor([ids] * args.num_samples, dtype=torch.long)
    out = model.generate(idx, args.new_tokens, temperature=args.temperature, top_k=args.top_k or None, rngs=args.seed)
    for i, row in enumerate(out.tolist()):
        print(f"--- sample {i} ---")
        print(tok.decode(row))


def sample_from_folder(args):
    """Continues token-id prompts (text prompts go through the byte / BPE tokenizer) with a model folder."""
    from jax_gpt_b200.models.registry import load_model
    device = "cuda" if torch.cuda.is_available() else "cpu"
    dtype = getattr(torch, args.dtype) if device == "cuda" else torch.float32
    family, cfg, params = load_model(args.model_dir, dtype, device)
    prompts = [[int(i) for i in p.split(",")] for p in args.prompt_ids] or [get_tokenizer().encode(args.prompt)] * args.num_samples
    bad = [i for p in prompts for i in p if not 0 <= i < cfg.vocab_size]
    if bad:
        sys.exit(f"token ids outside the vocabulary of {cfg.vocab_size}: {bad[:8]}")
    out = family.mod().generate(params, prompts, cfg, args.new_tokens, temperature=args.temperature, top_k=args.top_k or None, key=args.seed)
    for i, row in enumerate(out.tolist()):
        print(f"--- sample {i} ---")
        print(",".join(map(str, row)))


if __name__ == "__main__":
    main()
