"""What the model drivers share: one sequence at a time, its position on the device and on the host, greedy or sampled
next tokens, decode steps replayed from CUDA graphs, prompts in portions, generation.

A model supplies ``_step_ops(key)`` -- the operators of one decode step, reading ``self.token`` / ``self.cur_pos`` and
leaving ``self.logits`` -- and may replace ``prefill`` (by default a prompt goes through the decode step token by
token).  ``PortionDriver`` is the driver of the models that run a prompt in portions of many tokens."""

from __future__ import annotations

import torch

F32, I32, I64 = torch.float32, torch.int32, torch.int64
DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}
MAX_PORTION = 2048  # tokens of a prompt that run at once


class SequenceDriver:
    backend = "deepseek_v3_2"  # the native library whose sampling operator and status word the model uses

    def _init_sequence(self, device, vocab_local: int, use_graph: bool) -> None:
        dev = self.device = torch.device(device)
        self.cur_pos = torch.zeros(1, dtype=I32, device=dev)
        self.token = torch.zeros(1, dtype=I64, device=dev)
        self.logits = torch.zeros(1, 1, vocab_local, dtype=F32, device=dev)
        self.token_out = torch.zeros(1, dtype=I64, device=dev)
        self.use_graph = use_graph
        self._graphs: dict = {}
        # Host copy of the device-resident position: the kernels write cache row ``cur_pos`` and mask on it,
        # while the host picks a step's launch shapes from ``pos``; the two must not drift, and a position
        # past what the model can hold must be refused before anything is launched.
        self._pos = 0
        # sampling state (the reference's SAMPLING_CONFIG / TOP_P_SCORES / TOP_N_LOG_PROBS / TOP_N_INDICES
        # temp vars, temp_var_indices.py:64-73): greedy until set_sampling is called
        self.sampling_config = torch.tensor([0.0, 1.0, 0.0, 0.0], dtype=F32, device=dev)  # temperature, top_p, top_k, use_top_p
        self.sampling_seed = 0
        self.sampling = False
        self.sample_step = torch.zeros(2, dtype=I64, device=dev)  # advanced by every launch (graph replay safe)
        self.sampled = torch.zeros(1, dtype=I32, device=dev)
        self.token_logprob = torch.zeros(1, dtype=F32, device=dev)
        self.topn_logprobs = torch.zeros(1, 256, dtype=F32, device=dev)
        self.topn_indices = torch.zeros(1, 256, dtype=I32, device=dev)

    # -- what a model supplies --
    def position_limit(self) -> int:
        """Positions a sequence may reach (exclusive)."""
        raise NotImplementedError

    def _step_ops(self, key) -> None:
        raise NotImplementedError

    def _graph_key(self, pos: int):
        """Steps at positions with the same key have the same launches."""
        raise NotImplementedError

    def _sample_op(self):
        raise NotImplementedError

    # -- reference driver controls (end2end.py:551-577) --
    def reset_sequence(self) -> None:
        self.cur_pos.zero_()
        self._pos = 0

    def set_cur_pos(self, pos: int) -> None:
        if not 0 <= pos < self.position_limit():
            raise ValueError(f"set_cur_pos({pos}): a sequence holds {self.position_limit()} positions")
        self.cur_pos.fill_(pos)
        self._pos = pos

    def set_sampling(self, temperature: float = 0.0, top_p: float = 1.0, top_k: int = 0, use_top_p: bool = False,
                     seed: int | None = None) -> None:
        """Sample the next token instead of taking the arg-max (end2end.py:253-311: temperature, top-p, top-k
        per request; ``set_sampling_seed``).  Temperature 0 with no seed change returns to greedy decoding.
        The token's log-probability and the top-256 log-probabilities / ids are left in ``token_logprob``,
        ``topn_logprobs`` and ``topn_indices`` after every step."""
        self.sampling_config.copy_(torch.tensor([temperature, top_p, float(top_k), 1.0 if use_top_p else 0.0]))
        if seed is not None and seed != self.sampling_seed:
            self.sampling_seed = seed
            self._graphs.clear()  # the seed is a launch argument
        if not self.sampling:
            self.sampling = True
            self._graphs.clear()

    def set_sampling_seed(self, seed: int) -> None:
        """end2end.py:120-134."""
        if seed != self.sampling_seed:
            self.sampling_seed = seed
            self._graphs.clear()

    def _choose(self, logits: torch.Tensor) -> None:
        """The next token of ``logits`` [1, vocab] into ``token_out``."""
        if self.sampling:
            self._sample_op()(logits, self.sampling_config, self.sampled, seed=self.sampling_seed, step=self.sample_step,
                              token_logprob=self.token_logprob, topn_logprobs=self.topn_logprobs, topn_indices=self.topn_indices)
            self.token_out.copy_(self.sampled)
        else:
            self.token_out.copy_(torch.argmax(logits.view(-1)))

    # -- the step --
    def _may_capture(self) -> bool:
        return self.use_graph

    def _check_positions(self, what: str, pos: int, n: int) -> None:
        if pos != self._pos:
            raise ValueError(f"{what}: the device position is {self._pos} (use set_cur_pos to move it)")
        if pos + n > self.position_limit():
            raise ValueError(f"{what}: past the end of the {self.position_limit()} positions a sequence may have")

    def forward(self, token: int | torch.Tensor, pos: int) -> None:
        """Run one decode step for ``token`` at position ``pos`` (asynchronous; results in
        ``self.logits`` / ``self.token_out``)."""
        self._check_positions(f"forward(pos={pos})", pos, 1)
        if isinstance(token, int):
            self.token.fill_(token)
        else:
            self.token.copy_(token.view(-1)[:1])
        self._pos = pos + 1
        key = self._graph_key(pos)
        if not self._may_capture():
            self._step_ops(key)
            return
        if key not in self._graphs:
            saved, saved_step = self.cur_pos.clone(), self.sample_step.clone()
            self._step_ops(key)  # warm-up outside capture (lazy function attributes, allocator)
            torch.cuda.synchronize()
            self.cur_pos.copy_(saved)
            self.sample_step.copy_(saved_step)  # the warm-up drew a number: give it back
            g = torch.cuda.CUDAGraph()
            with torch.cuda.graph(g):
                self._step_ops(key)
            self.cur_pos.copy_(saved)
            self._graphs[key] = g
        self._graphs[key].replay()

    def prefill(self, tokens: list[int], want: list[int] | None = None) -> torch.Tensor:
        """Run the sequence's next ``tokens``; returns the f32 logits [len(want), vocab] at the places ``want`` among
        them (default: the last one) and leaves ``logits`` / ``token_out`` as a decode step of the last token would."""
        want = [len(tokens) - 1] if want is None else want
        rows: dict[int, torch.Tensor] = {}
        for i, tok in enumerate(tokens):
            self.forward(int(tok), self._pos)
            if i in want:
                rows[i] = self.logits.view(-1).clone()
        return torch.stack([rows[i] for i in want]) if want else self.logits.view(1, -1)[:0]

    @torch.no_grad()
    def generate(self, prompt: list[int], n_new: int, collect_logits: bool = False):
        """Prompt, then decoding (tilert/models/deepseek_v3_2/generator.py:187-265).
        Returns the generated tokens (and the f32 logits of each generated position)."""
        self.reset_sequence()
        self.prefill(prompt)
        pos = len(prompt)
        toks, lgs = [], []
        for i in range(n_new):
            if collect_logits:
                lgs.append(self.logits.view(-1).clone())
            nxt = self.token_out.clone()
            toks.append(nxt)
            if self.decode_past_last or i + 1 < n_new:
                self.forward(nxt, pos)
            pos += 1
        toks = [int(t) for t in torch.cat(toks).cpu()]
        return (toks, lgs) if collect_logits else toks

    decode_past_last = False  # run the last generated token through the model too


class PortionDriver(SequenceDriver):
    """Prompts in portions (``_prefill_portion``), decode steps whose launch shapes depend on a bound of the keys read."""

    portion: int        # most tokens of a prompt that run at once
    max_window: int     # most keys any layer attends to
    # filled by prompts when a caller asks for it: the residual after every layer run, [runs][tokens, dim] f32
    layer_taps: list[torch.Tensor] | None = None

    def _prefill_portion(self, tokens: list[int], want: list[int], last: bool) -> torch.Tensor:
        """One portion; f32 logits [len(want), vocab] of the wanted places; with ``last`` also those of the last token
        in ``self.logits``.  Advances the position."""
        raise NotImplementedError

    def _graph_key(self, pos: int) -> int:
        """A bound of the keys any layer attends to: a power of two, constant once every window is full."""
        n = 256
        while n < pos + 1 and n < self.max_window:
            n *= 2
        return n

    @torch.no_grad()
    def prefill(self, tokens: list[int], want: list[int] | None = None) -> torch.Tensor:
        self._check_positions("prefill", self._pos, len(tokens))
        if len(tokens) == 1:
            return super().prefill(tokens, want)  # the decode step is the faster form for one token
        outs = []
        for lo in range(0, len(tokens), self.portion):
            part = tokens[lo: lo + self.portion]
            here = [w - lo for w in (want if want is not None else []) if lo <= w < lo + len(part)]
            outs.append(self._prefill_portion(part, here, lo + len(part) == len(tokens)))
        self._choose(self.logits.view(1, -1))
        return self.logits.view(1, -1).clone() if want is None else torch.cat(outs)
