"""Small Rozesun configurations and the error measure shared by the tests of that design."""

import functools

import torch

from oracle import rozesun as R
from ralasun_models import row_errors
from tilert_b200 import synthetic
from tilert_b200.models.rozesun.model_args import LayerArgs, LoopArgs, MixerArgs, MlpArgs, RozesunArgs, toy_args


def _wide(heads, dim, rot, vdim, q_rank, kv_rank, scale, base=10000.0):
    return MixerArgs("latent_attention", heads, dim, rot, vdim, q_rank, kv_rank, scale, base)


def _near(heads, dim, rot, vdim, q_rank, kv_rank, scale, window, base=10000.0):
    return MixerArgs("latent_attention_2", heads, dim, rot, vdim, q_rank, kv_rank, scale, base, window)


def _uneven() -> RozesunArgs:
    """Sizes that are no multiples of eight, every layer with its own, the loop at the very beginning."""
    return RozesunArgs(vocab_size=301, dim=90, eps=3e-4, logit_scale=1.7, max_seq_len=400, loop=LoopArgs(0, 2, 3), layers=(
        LayerArgs(_near(3, 10, 6, 9, 27, 21, 0.41, 9, base=300.0), MlpArgs(35, 0.7)),
        LayerArgs(_wide(5, 22, 14, 30, 33, 45, 0.2, base=2000.0), MlpArgs(50, 3.0)),
        LayerArgs(_near(1, 7, 2, 5, 6, 5, 0.9, 24), None),
        LayerArgs(_near(7, 18, 10, 13, 50, 70, 0.25, 70, base=50.0), MlpArgs(35, 1.1))))


def _alike() -> RozesunArgs:
    """Sizes that usually differ are the same, no loop, many heads: tiles that hold rows of several heads and tokens."""
    m = MlpArgs(64, 1.0)
    return RozesunArgs(vocab_size=64, dim=64, eps=1e-6, logit_scale=1.0, max_seq_len=420, layers=(
        LayerArgs(_wide(20, 16, 16, 16, 16, 16, 0.3), m), LayerArgs(_near(20, 16, 16, 16, 16, 16, 0.3, 16), m)))


def _deep() -> RozesunArgs:
    """A wide latent, small heads (the expanded form pays early), the loop at the end, one pass, sharp scores."""
    return RozesunArgs(vocab_size=640, dim=128, eps=1e-5, logit_scale=0.3, max_seq_len=420, loop=LoopArgs(1, 3, 1), layers=(
        LayerArgs(_near(4, 24, 40, 72, 96, 272, 0.2, 40), MlpArgs(160, 1.0)), LayerArgs(_wide(3, 64, 32, 64, 48, 320, 0.2), None),
        LayerArgs(_near(4, 24, 40, 72, 96, 272, 0.2, 130), MlpArgs(160, 4.0))))


def _one() -> RozesunArgs:
    """Windows of one and of two positions, one head, the whole model looped."""
    return RozesunArgs(vocab_size=50, dim=32, eps=1e-6, logit_scale=1.0, max_seq_len=128, loop=LoopArgs(0, 2, 2), layers=(
        LayerArgs(_near(2, 8, 8, 16, 16, 16, 0.35, 1), MlpArgs(16, 2.0)), LayerArgs(_near(1, 8, 4, 8, 8, 24, 0.35, 2), MlpArgs(24, 2.0))))


CONFIGS = {"toy": lambda: toy_args(400), "uneven": _uneven, "alike": _alike, "deep": _deep, "one": _one}


@functools.lru_cache(maxsize=None)
def case(name: str, n: int, seed: int = 0):
    """(args, weights, tokens, exact logits [n, vocab], residual after every layer run)."""
    args = CONFIGS[name]()
    sd = synthetic.random_rozesun_state_dict(args, seed=7)
    toks = torch.randint(0, args.vocab_size, (n,), generator=torch.Generator().manual_seed(seed)).tolist()
    taps: list = []
    ref = R.forward(args.to_config(), sd, toks, torch.float64, taps)
    return args, sd, toks, ref, taps


LIMITS = {"float32": (2e-5, 2e-6), "bfloat16": (5e-2, 2e-2)}  # worst row, median row


def check_rows(what: str, dtype: str, ref: torch.Tensor, out: torch.Tensor) -> None:
    assert out.shape == ref.shape, (what, out.shape, ref.shape)
    e = row_errors(ref, out)
    worst, median = LIMITS[dtype]
    over = torch.nonzero(e > worst).flatten().tolist()
    assert not over and float(e.median()) <= median, \
        f"{what} {dtype}: {len(over)} of {len(e)} rows over, first {over[:5]}, worst {float(e.max()):.2e}, median {float(e.median()):.2e}"
    assert bool(torch.isfinite(out).all())
