"""Whole-model driver of a Ralasun decoder: embedding and its norm, the layers, the final norm and the head, on the
shared sequence driver (positions, sampling, graph replay, generation)."""

from __future__ import annotations

import torch

from tilert_b200 import gqa_ops as ops
from tilert_b200.gqa_ops import F32, I32, I64, pad

from ..blocks import Scratch, Stream, one_plus, padded_rows
from ..driver import DTYPES, MAX_PORTION, PortionDriver
from .layer import LayerWeights, RalasunLayer
from .model_args import RalasunArgs


class RalasunModel(PortionDriver):
    backend = "ralasun"

    def __init__(self, args: RalasunArgs, sd, device="cuda", dtype: str = "bfloat16", use_graph: bool = True,
                 portion: int | None = None):
        """``sd``: checkpoint tensors by name.  ``dtype``: type of activations and caches; ``float32`` makes every
        product true 32-bit arithmetic.  ``portion``: most tokens of a prompt that run at once."""
        self.args, self.dtype = args, DTYPES[dtype]
        dev = torch.device(device)
        if dev.type == "cuda" and dev.index is None:
            dev = torch.device("cuda", torch.cuda.current_device())
        self.portion = min(portion or MAX_PORTION, args.max_seq_len)
        self.embed = padded_rows(sd["embed"], dev)
        self.embed_norm, self.final_norm = one_plus(sd["embed.norm"], dev), one_plus(sd["final.norm"], dev)
        self.head = padded_rows(sd["head"], dev)
        for name, t in (("embed", self.embed), ("head", self.head)):
            if tuple(t.shape) != (args.vocab_size, pad(args.dim)):
                raise ValueError(f"{name} has shape {tuple(t.shape)}, the configuration says {args.vocab_size} x {args.dim}")
        self.scratch = Scratch(dev)
        self.layers: list[RalasunLayer] = []
        mixed = False
        for li, a in enumerate(args.layers):
            v_mode = ops.VMIX_NONE if not a.mixer.v_mix else (ops.VMIX_BLEND if mixed else ops.VMIX_FIRST)
            mixed = mixed or a.mixer.v_mix
            self.layers.append(RalasunLayer(args, li, LayerWeights(args, sd, li, dev), self.scratch, self.portion, self.dtype, dev, v_mode))
        self._init_sequence(dev, args.vocab_size, use_graph)
        self.max_window = max(layer.cache.visible(args.max_seq_len) for layer in self.layers) if self.layers else 1

    @classmethod
    def from_pretrained(cls, model_dir, device="cuda", dtype: str = "bfloat16", max_seq_len: int | None = None, **kw) -> "RalasunModel":
        """``config.json`` and ``*.safetensors`` of a directory."""
        from tilert_b200.convert import HFCheckpoint

        return cls(RalasunArgs.from_dir(model_dir, max_seq_len), HFCheckpoint(model_dir), device, dtype, **kw)

    def position_limit(self) -> int:
        return self.args.max_seq_len

    def weight_bytes(self) -> int:
        """Bytes of weights one decode step streams (head included, one embedding row not)."""
        return sum(layer.w.weight_bytes(layer.a) for layer in self.layers) + 2 * self.head.numel()

    # -- one token --
    def _step_ops(self, length: int) -> None:
        a = self.args
        st = Stream(self.scratch, a.dim)
        ops.embed_norm(self.token, self.embed, self.embed_norm, a.eps, a.dim, st.x.view(1, -1))
        for layer in self.layers:
            layer.decode(st, self.cur_pos, length)
        st.dense(self.head, self.logits, a.vocab_size, a.dim, a.eps, gain2=self.final_norm)
        self._choose(self.logits.view(1, -1))
        self.cur_pos += 1

    def _sample_op(self):
        return ops.sample

    # -- prompts --
    def _prefill_portion(self, tokens: list[int], want: list[int], last: bool) -> torch.Tensor:
        a, sc, n = self.args, self.scratch, len(tokens)
        ids = torch.tensor(tokens, dtype=I64).to(self.device)
        x, xh = sc.get("x", self.portion, pad(a.dim)), sc.get("xh", self.portion, pad(a.dim), dtype=self.dtype)
        ops.embed_norm(ids, self.embed, self.embed_norm, a.eps, a.dim, x, xh)
        for layer in self.layers:
            layer.prefill(x, xh, n, self.cur_pos)
            if self.layer_taps is not None:
                self.layer_taps.append(x[:n, : a.dim].clone())
        out = torch.empty(len(want), a.vocab_size, dtype=F32, device=self.device)
        if want:
            rows = torch.tensor(want, dtype=I32).to(self.device)
            xn = torch.zeros(len(want), pad(a.dim), dtype=self.dtype, device=self.device)
            ops.gather_norm(x, rows, self.final_norm, a.eps, a.dim, xn)
            ops.gemm(xn, self.head, out, len(want), a.vocab_size, a.dim)
        if last:
            ops.vec_dense(x[n - 1], self.head, self.logits, a.vocab_size, a.dim, gain2=self.final_norm, eps=a.eps)
        self.cur_pos += n
        self._pos += n
        return out
