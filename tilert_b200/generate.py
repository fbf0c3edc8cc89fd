"""``python -m tilert_b200.generate``: the reference's text-generation entry (tilert/generate.py:75-150) for
this backend.  No checkpoint or tokenizer ships with the repository, so the runnable form is
``--use-random-weights`` with a seeded random prompt of ``--prompt-len`` token ids (the reference's own
``prompt_tokens=`` path, generator.py:160,195).

    python -m tilert_b200.generate --model toy --use-random-weights --max-new-tokens 32 [--with-mtp]
    python -m tilert_b200.generate --model ralasun --use-random-weights [--dtype float32]   # likewise --model rozesun
    python -m tilert_b200.generate --model-weights-dir DIR      # the family is chosen by DIR/config.json
"""

from __future__ import annotations

import argparse
import statistics

import torch

from tilert_b200.models import registry


def parse_args():
    ap = argparse.ArgumentParser(description=__doc__.split("\n")[0])
    ap.add_argument("--model", default="toy", choices=registry.presets(),
                    help="toy: the 2-layer test model; deepseek_v3_2: the full shape with --layers layers; ralasun, rozesun: "
                         "a small model of that design")
    ap.add_argument("--dtype", default="bfloat16", help="activation type of a family that runs in more than one")
    ap.add_argument("--layers", type=int, default=2, help="decoder layers of the full-shape model (61 in the real one)")
    ap.add_argument("--use-random-weights", action="store_true")
    ap.add_argument("--model-weights-dir", default=None, help="checkpoint directory: config.json and *.safetensors")
    ap.add_argument("--with-mtp", action="store_true")
    ap.add_argument("--max-new-tokens", type=int, default=32)
    ap.add_argument("--prompt-len", type=int, default=16)
    ap.add_argument("--max-seq-len", type=int, default=1024)
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--seed", type=int, default=0)
    return ap.parse_args()


def main() -> None:
    args = parse_args()
    import tilert_b200

    if not torch.cuda.is_available():
        raise SystemExit("tilert_b200.generate needs a CUDA device (sm_100a); there is no CPU path")
    weights_dir = None if args.use_random_weights else args.model_weights_dir
    family = registry.family_of_preset(args.model) if weights_dir is None else registry.family_of_dir(weights_dir)
    if args.dtype not in family.dtypes:
        raise SystemExit(f"{family.name} runs in {', '.join(family.dtypes)}, not in {args.dtype}")
    if args.with_mtp and family.name != "deepseek_v3_2":
        raise SystemExit(f"{family.name} has no multi-token prediction layer")
    tilert_b200.load_backend(family.backend)
    tilert_b200.tilert_init(0, family.backend)
    gen = family.generator(weights_dir, args)
    if args.temperature > 0:
        gen.update_sampling_config(args.temperature, args.top_p, args.top_k, args.top_p < 1.0)
    g = torch.Generator().manual_seed(args.seed + 1)
    prompt = torch.randint(0, gen.vocab_size(), (args.prompt_len,), generator=g).tolist()
    text, times, accepted, plen = gen.generate("", print_log=True, prompt_tokens=prompt)
    decode = times[-len(accepted):] if args.with_mtp else times[gen.prompt_steps(plen):]
    if decode:
        per_step = statistics.median(decode)
        toks = (sum(accepted) / len(accepted)) if accepted else 1.0
        print(f"prompt {plen} tokens, {len(decode)} decode steps, median {per_step * 1e3:.3f} ms per step, "
              f"{toks / per_step:.1f} tokens/s" + (f", mean accepted {toks:.2f}" if accepted else ""))
    gen.cleanup()


if __name__ == "__main__":
    main()
