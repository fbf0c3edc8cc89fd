"""Single-sequence generation: what the model families' generators share (tilert/models/deepseek_v3_2/generator.py:
155-265) -- prompt, per-step wall-clock times, end-of-sequence, printing.  A tokenizer is optional (none ships with this
repository): without one, prompts are token id lists and the returned text is the space-joined ids."""

from __future__ import annotations

import time

import torch


class SequenceGenerator:
    tokenizer = None
    eos_id = -1
    max_new_tokens = 100

    # -- what a family supplies --
    def _max_len(self) -> int:
        raise NotImplementedError

    def _prompt(self, tokens: list[int], times: list[float]) -> int:
        """Run the prompt, append the seconds of every step taken, return the next token."""
        raise NotImplementedError

    def _next(self, token: int) -> int:
        """One decode step."""
        raise NotImplementedError

    def _end_sequence(self) -> None:
        raise NotImplementedError

    def vocab_size(self) -> int:
        raise NotImplementedError

    def prompt_steps(self, prompt_len: int) -> int:
        """Entries of the times list that belong to a prompt of ``prompt_len`` tokens."""
        return prompt_len

    def _tokens_of(self, prompt, prompt_tokens):
        if prompt_tokens is not None:
            return list(prompt_tokens)
        if self.tokenizer is None:
            raise ValueError("no tokenizer: pass prompt_tokens=[...]")
        return self.tokenizer.apply_chat_template([{"role": "user", "content": prompt}], add_generation_prompt=True)

    def _text_of(self, toks: list[int]) -> str:
        if self.tokenizer is not None:
            return self.tokenizer.decode(toks, skip_special_tokens=True)
        return " ".join(str(t) for t in toks)

    def _generate_plain(self, prompt_tokens: list[int], print_log: bool):
        """(text, per-step seconds, [], prompt length); generator.py:187-265."""
        plen = len(prompt_tokens)
        total = min(self._max_len(), self.max_new_tokens + plen)
        times: list[float] = []
        out: list[int] = []
        nxt = self._prompt(prompt_tokens, times) if total > plen else None
        while plen + len(out) < total:
            out.append(nxt)
            if print_log:
                print(self._text_of([nxt]), end=" ", flush=True)
            if nxt == self.eos_id or plen + len(out) >= total:
                break
            t0 = time.time()
            nxt = self._next(nxt)
            times.append(time.time() - t0)
        self._end_sequence()
        if self.eos_id in out:
            out = out[: out.index(self.eos_id)]
        if print_log:
            print()
        return self._text_of(out) + "\n", times, [], plen


class PortionGenerator(SequenceGenerator):
    """Generation with a model on the ``PortionDriver``: prompts in portions, then graph-replayed steps."""

    def __init__(self, model, max_new_tokens: int = 100, tokenizer=None, eos_id: int = -1, sampling_seed: int = 0):
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
