"""Whole-model driver of a Rozesun decoder: embedding, the layers in the order of their runs (a block of them several times,
each pass with its own caches), the final norm and the tied head, on the shared driver of prompts in portions."""

from __future__ import annotations

import torch

from tilert_b200 import gqa_ops as ops
from tilert_b200.gqa_ops import BF16, F32, I32, I64, pad

from ..blocks import RowStream, Scratch, Stream, layer_norm, padded_rows, padded_vec
from ..driver import DTYPES, MAX_PORTION, PortionDriver
from .layer import LayerWeights, RozesunLayer
from .model_args import RozesunArgs


class RozesunModel(PortionDriver):
    backend = "ralasun"

    def __init__(self, args: RozesunArgs, sd, device="cuda", dtype: str = "bfloat16", use_graph: bool = True, portion: int | None = None):
        """``sd``: checkpoint tensors by name.  ``dtype``: type of activations and caches; ``float32`` makes every
        product true 32-bit arithmetic.  ``portion``: most tokens of a prompt that run at once."""
        self.args, self.dtype = args, DTYPES[dtype]
        dev = torch.device(device)
        if dev.type == "cuda" and dev.index is None:
            dev = torch.device("cuda", torch.cuda.current_device())
        self.portion = min(portion or MAX_PORTION, args.max_seq_len)
        self.embed = padded_rows(sd["embed"], dev)
        if tuple(self.embed.shape) != (args.vocab_size, pad(args.dim)):
            raise ValueError(f"embed has shape {tuple(self.embed.shape)}, the configuration says {args.vocab_size} x {args.dim}")
        self.final_norm = layer_norm(sd, "final.norm", dev, scale=args.logit_scale)  # the logits are linear in its result
        steps = None
        if args.loop is not None:
            steps = sd["loop.step"]
            if tuple(steps.shape) != (args.loop.times, args.dim):
                raise ValueError(f"loop.step has shape {tuple(steps.shape)}, the configuration says {args.loop.times} x {args.dim}")
        self.scratch = Scratch(dev)
        order = [li for li, _ in args.runs()]
        ropes: dict = {}
        self.layers: list[RozesunLayer] = []
        for li, a in enumerate(args.layers):
            m = a.mixer
            key = (m.rot_base, m.rot_dim)
            if key not in ropes:
                ropes[key] = ops.rotation_table(m.rot_base, m.rot_dim, args.max_seq_len, dev)
            weights = LayerWeights(args, sd, li, dev, expanded=self.dtype == BF16 and ops.expanded_fits(m))
            self.layers.append(RozesunLayer(args, li, weights, ops.Rotation(ropes[key], m.interleaved), self.scratch, self.portion,
                                            self.dtype, dev, order.count(li)))
        # (layer, its pass, vector added to the residual in front of it or None)
        self.runs: list[tuple[RozesunLayer, int, torch.Tensor | None]] = []
        done = [0] * len(args.layers)
        for li, begins in args.runs():
            self.runs.append((self.layers[li], done[li], None if begins is None else padded_vec(steps[begins], dev)))
            done[li] += 1
        self._init_sequence(dev, args.vocab_size, use_graph)
        self.max_window = max((c.visible(args.max_seq_len) for layer in self.layers for c in layer.caches), default=1)

    @classmethod
    def from_pretrained(cls, model_dir, device="cuda", dtype: str = "bfloat16", max_seq_len: int | None = None, **kw) -> "RozesunModel":
        """``config.json`` and ``*.safetensors`` of a directory."""
        from tilert_b200.convert import HFCheckpoint

        return cls(RozesunArgs.from_dir(model_dir, max_seq_len), HFCheckpoint(model_dir), device, dtype, **kw)

    def position_limit(self) -> int:
        return self.args.max_seq_len

    def weight_bytes(self) -> int:
        """Bytes of weights one decode step streams (a looped layer's in every pass; the head, but not an embedding row)."""
        return sum(layer.weight_bytes() for layer in self.layers) + 2 * self.embed.numel()

    # -- one token --
    def _step_ops(self, length: int) -> None:
        a = self.args
        st = Stream(self.scratch, a.dim)
        ops.embed_norm(self.token, self.embed, None, a.eps, a.dim, st.x.view(1, -1))
        for layer, nr, add in self.runs:
            st.add = add
            layer.decode(st, nr, self.cur_pos, length)
        st.dense(self.embed, self.logits, a.vocab_size, a.dim, a.eps, gain2=self.final_norm)
        self._choose(self.logits.view(1, -1))
        self.cur_pos += 1

    def _sample_op(self):
        return ops.sample

    # -- prompts --
    def _prefill_portion(self, tokens: list[int], want: list[int], last: bool) -> torch.Tensor:
        a, sc, n = self.args, self.scratch, len(tokens)
        ids = torch.tensor(tokens, dtype=I64).to(self.device)
        st = RowStream(sc.get("x", self.portion, pad(a.dim)), sc.get("xh", self.portion, pad(a.dim), dtype=self.dtype), n, a.dim, a.eps)
        ops.embed_norm(ids, self.embed, None, a.eps, a.dim, st.x)
        for layer, nr, add in self.runs:
            st.add = add
            layer.prefill(st, nr, self.cur_pos, self._pos)
            if self.layer_taps is not None:
                self.layer_taps.append(st.settle()[:n, : a.dim].clone())
        x = st.settle()
        out = torch.empty(len(want), a.vocab_size, dtype=F32, device=self.device)
        if want:
            rows = torch.tensor(want, dtype=I32).to(self.device)
            xn = torch.zeros(len(want), pad(a.dim), dtype=self.dtype, device=self.device)
            ops.gather_norm(x, rows, self.final_norm, a.eps, a.dim, xn)
            ops.gemm(xn, self.embed, out, len(want), a.vocab_size, a.dim)
        if last:
            ops.vec_dense(x[n - 1], self.embed, self.logits, a.vocab_size, a.dim, gain2=self.final_norm, eps=a.eps)
        self.cur_pos += n
        self._pos += n
        return out
