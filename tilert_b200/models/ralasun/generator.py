"""Generation with a Ralasun model through the shared generator: prompts in portions, then graph-replayed steps."""

from __future__ import annotations

import time

import torch

from ..generator import SequenceGenerator
from .model import RalasunModel


class RalasunGenerator(SequenceGenerator):
    def __init__(self, model: RalasunModel, max_new_tokens: int = 100, tokenizer=None, eos_id: int = -1, sampling_seed: int = 0):
        self.model, self.max_new_tokens = model, max_new_tokens
        self.tokenizer, self.eos_id, self.sampling_seed = tokenizer, eos_id, sampling_seed

    def update_sampling_config(self, temperature=0.0, top_p=1.0, top_k=0, use_topp=False) -> None:
        self.model.set_sampling(temperature, top_p, top_k, use_topp)

    @torch.inference_mode()
    def generate(self, prompt: str = "", print_log: bool = True, prompt_tokens: list[int] | None = None):
        """(text, seconds of the prompt's portions and of every step, [], prompt length)."""
        self.model.set_sampling_seed(self.sampling_seed)
        self.model.reset_sequence()
        return self._generate_plain(self._tokens_of(prompt, prompt_tokens), print_log)

    def _max_len(self) -> int:
        return self.model.position_limit()

    def _prompt(self, tokens: list[int], times: list[float]) -> int:
        for lo in range(0, len(tokens), self.model.portion):
            t0 = time.time()
            self.model.prefill(tokens[lo: lo + self.model.portion])
            nxt = int(self.model.token_out)
            times.append(time.time() - t0)
        return nxt

    def _next(self, token: int) -> int:
        self.model.forward(token, self.model._pos)
        return int(self.model.token_out)

    def vocab_size(self) -> int:
        return self.model.args.vocab_size

    def prompt_steps(self, prompt_len: int) -> int:
        return -(-prompt_len // self.model.portion)

    def _end_sequence(self) -> None:
        self.model.reset_sequence()

    def cleanup(self) -> None:
        torch.cuda.synchronize()
