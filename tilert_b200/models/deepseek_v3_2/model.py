"""Whole-model driver for batch-1 greedy decoding: embedding lookup, the decoder layers, the
vocabulary head and arg-max -- the role of the reference's ``ShowHandsDSALayer``
(tilert/models/deepseek_v3_2/modules/end2end.py:166-703) whose forward is one native call per
token.  Here a step is the layers' operator sequence, replayed from a CUDA graph."""

from __future__ import annotations

import torch

from ..driver import SequenceDriver
from . import ops
from .layer import DecoderLayer, LayerScratch, LayerWeights, precompute_freqs
from .model_args import ModelArgs

BF16 = torch.bfloat16
F32 = torch.float32
I32 = torch.int32


class DsaModel(SequenceDriver):
    decode_past_last = True  # (the caches then hold every generated token, as the reference's loop leaves them)

    def __init__(self, args: ModelArgs, sd: dict[str, torch.Tensor], device="cuda", cache_len: int | None = None,
                 world: int = 1, rank: int = 0, comm: int | None = None, use_graph: bool = True,
                 share_scratch: bool | None = None, temp_vars: list[torch.Tensor] | None = None):
        """``share_scratch``: one scratch set for all layers instead of one per layer (default: when the model
        has more than four layers).  ``temp_vars``: the reference driver's list of 56 scratch tensors
        (``DsaTempVarIdx``); the layers' scratch, the logits and the output token then live in it."""
        self.args, self.device = args, torch.device(device)
        self.world, self.rank, self.comm = world, rank, comm
        dev = self.device
        self.cache_len = cache_len or args.max_seq_len
        v_l = args.vocab_size // world
        if args.vocab_size % world != 0:
            raise ValueError(f"vocab_size {args.vocab_size} does not divide over {world} ranks")
        packed = sd if isinstance(sd, dict) and "layers" in sd else None  # a converted model (convert.load_model)
        if packed is not None:
            if packed["world"] != world:
                raise ValueError(f"the converted weights were sharded for {packed['world']} ranks, not {world}")
            self.embed, self.final_norm, self.head = packed["embed"], packed["final_norm"], packed["head"]
            layer_weights = packed["layers"]
        else:
            self.embed = sd["model.embed_tokens.weight"].to(dev, BF16)
            self.final_norm = sd["model.norm.weight"].to(dev, F32)
            self.head = sd["lm_head.weight"][rank * v_l:(rank + 1) * v_l].to(dev, BF16).contiguous()
            layer_weights = None
        if share_scratch is None:
            share_scratch = args.n_layers > 4 or temp_vars is not None
        scratch = None
        if temp_vars is not None:
            scratch = LayerScratch.from_temp_vars(args, temp_vars, self.cache_len, 1, world)
        elif share_scratch:
            scratch = LayerScratch(args, dev, self.cache_len, 1, world)
        self.layers = [
            DecoderLayer(args, layer_weights[li] if layer_weights is not None else LayerWeights(args, sd, li, dev, world, rank),
                         dev, self.cache_len, 1, world, comm, scratch=scratch, out_slot=li)
            for li in range(args.n_layers)
        ]
        self.freqs = precompute_freqs(args).to(dev)
        self._init_sequence(dev, v_l, use_graph)
        self.full_logits: torch.Tensor | None = None  # world > 1 and sampling: every rank's slice, gathered
        self.temp_vars = temp_vars
        if temp_vars is not None:
            from .temp_var_indices import Idx

            self.logits = temp_vars[Idx.LOGITS_OUT].reshape(-1)[:v_l].view(1, 1, v_l)
            self.cur_pos = temp_vars[Idx.CUR_POS].reshape(-1)[:1]

    @classmethod
    def from_converted(cls, args: ModelArgs, out_dir, device="cuda", rank: int = 0, **kw) -> "DsaModel":
        """A model on the per-rank packed files that ``python -m tilert_b200.convert`` wrote."""
        from tilert_b200 import convert

        packed = convert.load_model(out_dir, device, rank)
        return cls(args, packed, device, world=packed["world"], rank=rank, **kw)

    def position_limit(self) -> int:
        return min(self.cache_len, self.freqs.shape[0])  # rows of the caches, positions of the rotary table

    def set_sampling(self, temperature: float = 0.0, top_p: float = 1.0, top_k: int = 0, use_top_p: bool = False,
                     seed: int | None = None) -> None:
        if self.world > 1:
            import torch.distributed as dist

            if not (dist.is_available() and dist.is_initialized()):
                raise ValueError("sampling over a vocabulary split across ranks gathers the logits with "
                                 "torch.distributed: initialise the default process group first")
            if self.full_logits is None:
                self.full_logits = torch.zeros(self.args.vocab_size, dtype=F32, device=self.device)
        super().set_sampling(temperature, top_p, top_k, use_top_p, seed)

    def inject_cache(self, layer_caches, start_pos: int = 0, end_pos: int | None = None) -> None:
        """``layer_caches``: one (ki, kv, pe) bf16 triple per layer from an external prefill
        (DSAv32Generator.inject_cache, generator.py:419-484); follow with ``set_cur_pos``.  A triple of
        uint8 planes (kv_raw [seq, 528], pe_raw [seq, 128], ki_pages [pages, 8448]) is taken as the FP8 wire
        format of pd_vllm/profiles/mla_nsa.py and needs ``end_pos`` (the pages do not tell the length)."""
        for layer, (c0, c1, c2) in zip(self.layers, layer_caches):
            if c0.dtype == torch.uint8:
                if end_pos is None:
                    raise ValueError("inject_cache: end_pos is needed with FP8 planes")
                layer.inject_cache_fp8(c0, c1, c2, end_pos - start_pos, start_pos)
            else:
                n = c0.shape[0] if end_pos is None else end_pos - start_pos
                layer.inject_cache(c0[:n], c1[:n], c2[:n], start_pos)

    def _step_ops(self, n_keys: int) -> None:
        x = self.embed[self.token].view(1, 1, -1)
        fr = self.freqs[self.cur_pos.long()]
        for layer in self.layers:
            x = layer.forward(x, self.cur_pos, fr, n_keys)
        ops.rmsnorm_head_proj(x, self.final_norm, self.head, None, self.logits, eps=self.args.eps)
        if self.world > 1 and self.sampling:
            # every rank gathers all slices of the logits (517 KB) and draws the same token: same seed, same step
            import torch.distributed as dist

            dist.all_gather_into_tensor(self.full_logits, self.logits.view(-1))
            ops.sample(self.full_logits.view(1, -1), self.sampling_config, self.sampled, seed=self.sampling_seed,
                       step=self.sample_step, token_logprob=self.token_logprob, topn_logprobs=self.topn_logprobs,
                       topn_indices=self.topn_indices)
            self.token_out.copy_(self.sampled)
        elif self.world > 1:
            # every rank holds vocab / world rows of the head: exchange (value, index) pairs over peer memory
            ops.argmax_exchange(self.logits, self.rank * self.logits.shape[-1], self.token_out, comm=self.comm)
        else:
            self._choose(self.logits.view(1, -1))
        if self.temp_vars is not None:
            from .temp_var_indices import Idx

            self.temp_vars[Idx.TOKEN_OUT].view(-1)[:1].copy_(self.token_out)
            self.temp_vars[Idx.TOKEN_ID].view(-1)[:1].copy_(self.token)
        self.cur_pos += 1

    def _graph_key(self, pos: int) -> int:
        """Indexer scan length: next multiple of 256 above the position, so graphs are reused."""
        return min(self.cache_len, (pos // 256 + 1) * 256)

    def _sample_op(self):
        return ops.sample

    def _may_capture(self) -> bool:
        return self.use_graph and not (self.sampling and self.world > 1)  # the gather is a library collective: not captured
