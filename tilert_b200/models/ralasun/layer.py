"""Weights, caches and the operator sequence of one Ralasun layer.

A layer norms its sublayers' OUTPUTS: x += n1(attention(x)), x += n2(experts(x)), and the sublayers read the residual
itself.  Two forms of the same layer:

* ``decode`` -- one token, f32 vectors.  The norm and the residual step behind a sublayer need the whole output
  vector, so they ride on the NEXT launch's input staging (``Pending``): six launches per layer -- qkv product, q/k
  norms + value mix + cache write + attention, output product, router, gate/up with routing, down.
* ``prefill`` -- a portion of tokens, activations in bf16 (or f32 in the exact mode), products on the tensor cores,
  experts as grouped products over the rows sorted by expert.
"""

from __future__ import annotations

import torch

from tilert_b200 import gqa_ops as ops
from tilert_b200.gqa_ops import BF16, F32, I32, pad
from tilert_b200.kv_cache import RingKVCache

from ..blocks import Pending, Scratch, Stream, one_plus, padded_rows
from .model_args import GATE_ALPHA, LayerArgs, RalasunArgs


class LayerWeights:
    """One layer's tensors, read under their checkpoint names from ``sd`` (any key -> tensor mapping)."""

    def __init__(self, args: RalasunArgs, sd, li: int, device):
        a = args.layers[li]
        dev = torch.device(device)
        mix, mlp = f"l{li}.mix", f"l{li}.mlp"
        self.qkv = padded_rows(torch.cat([sd[f"{mix}.{n}"].to(dev) for n in ("q", "k", "v")]), dev)
        self.q_gain = sd[f"{mix}.q.norm"].to(dev, F32).contiguous()
        self.k_gain = sd[f"{mix}.k.norm"].to(dev, F32).contiguous()
        self.lam = sd[f"{mix}.vmix"].to(dev, F32).reshape(1) if a.mixer.v_mix and f"{mix}.vmix" in sd else None
        self.o = padded_rows(sd[f"{mix}.o"], dev)
        self.norm1 = one_plus(sd[f"l{li}.norm1"], dev)
        self.norm2 = self.router = self.router_bias = self.gate_up = self.down = None
        self.shared_gate_up = self.shared_down = None
        if a.mlp is None:
            return
        self.norm2 = one_plus(sd[f"l{li}.norm2"], dev)
        self.router = padded_rows(sd[f"{mlp}.router"], dev)
        self.router_bias = sd[f"{mlp}.router.b"].to(dev, F32).contiguous()

        def halves(p):
            return padded_rows(torch.stack([sd[f"{p}.gate"].to(dev), sd[f"{p}.up"].to(dev)]), dev)

        e0 = halves(f"{mlp}.e0")
        self.gate_up = torch.empty(a.mlp.experts, *e0.shape, dtype=BF16, device=dev)       # [E, 2, ff, pad8(dim)]
        self.down = torch.empty(a.mlp.experts, args.dim, pad(a.mlp.ff), dtype=BF16, device=dev)
        for e in range(a.mlp.experts):
            self.gate_up[e] = e0 if e == 0 else halves(f"{mlp}.e{e}")
            self.down[e] = padded_rows(sd[f"{mlp}.e{e}.down"], dev)
        if a.mlp.shared_ff:
            self.shared_gate_up = halves(f"{mlp}.shared")
            self.shared_down = padded_rows(sd[f"{mlp}.shared.down"], dev)
        self._check(args, li)

    def _check(self, args: RalasunArgs, li: int) -> None:
        m, f = args.layers[li].mixer, args.layers[li].mlp
        want = {"qkv": (m.heads * m.dim + m.kv_heads * (m.dim + m.vdim), pad(args.dim)), "o": (args.dim, pad(m.heads * m.vdim)),
                "router": (f.experts, pad(args.dim)), "gate_up": (f.experts, 2, f.ff, pad(args.dim))}
        for name, shape in want.items():
            if tuple(getattr(self, name).shape) != shape:
                raise ValueError(f"layer {li}: {name} has shape {tuple(getattr(self, name).shape)}, the configuration says {shape}")

    def weight_bytes(self, args: LayerArgs) -> int:
        """Bytes of weights one decode step streams from HBM."""
        n = self.qkv.numel() + self.o.numel()
        if args.mlp is not None:
            n += self.router.numel() + args.mlp.top * (self.gate_up[0].numel() + self.down[0].numel())
            if self.shared_gate_up is not None:
                n += self.shared_gate_up.numel() + self.shared_down.numel()
        return 2 * n


class RalasunLayer:
    def __init__(self, args: RalasunArgs, li: int, weights: LayerWeights, scratch: Scratch, portion: int, dtype, device,
                 v_mode: int):
        self.args, self.a, self.w, self.sc = args, args.layers[li], weights, scratch
        self.dtype, self.portion, self.v_mode = dtype, portion, v_mode
        if v_mode == ops.VMIX_BLEND and weights.lam is None:
            raise ValueError(f"layer {li}: the weights have no value-mixing factor")
        m = self.a.mixer
        self.cache = RingKVCache(m.kv_heads, m.dim, m.vdim, m.window, args.max_seq_len, portion, device, dtype)
        self.n_q, self.n_kv = m.heads * m.dim, m.kv_heads * (m.dim + m.vdim)
        self.head_blocks = ops.head_blocks(m.heads, m.kv_heads)
        self.max_splits = max(1, 2 * ops.num_sms(device) // self.head_blocks)  # (two thread blocks per SM)

    def _v_first(self, rows: int):
        """Values of the first mixing layer, [rows, kv_heads * vdim] (all mixing layers agree on the size)."""
        if self.v_mode == ops.VMIX_NONE:
            return None
        return self.sc.get("v_first", rows, self.a.mixer.kv_heads * self.a.mixer.vdim)

    # -- one token --
    def decode(self, st: Stream, cur_pos: torch.Tensor, length: int) -> None:
        """``length``: an upper bound of the sequence's length including this token (sizes the key split)."""
        m, w, sc, eps, dim = self.a.mixer, self.w, self.sc, self.args.eps, self.args.dim
        qkv = sc.get("vec_qkv", pad(self.n_q + self.n_kv))
        st.dense(w.qkv, qkv, self.n_q + self.n_kv, dim, eps)
        n_splits = min(self.max_splits, (self.cache.visible(length) + 63) // 64)
        part = sc.get("vec_part", m.heads * n_splits * (pad(m.vdim, 16) + 2)) if n_splits > 1 else None
        counter = sc.get("vec_counter", self.head_blocks, dtype=I32) if n_splits > 1 else None
        att = sc.get("vec_att", pad(m.heads * m.vdim))
        ops.vec_attn(qkv, w.q_gain, w.k_gain, eps, self.v_mode, w.lam, self._v_first(1), m, self.cache, cur_pos, n_splits, part,
                     counter, att)
        y = sc.get("vec_y", pad(dim))
        ops.vec_dense(att, w.o, y, dim, m.heads * m.vdim)
        st.pending = Pending(y, w.norm1)
        f = self.a.mlp
        if f is None:
            return
        logits = sc.get("vec_router", pad(f.experts))
        st.dense(w.router, logits, f.experts, dim, eps, bias=w.router_bias)
        hidden = sc.get("vec_hidden", pad(f.shared_ff) + f.top * pad(f.ff), dtype=F32)
        ids, sw = sc.get("vec_ids", f.top, dtype=I32), sc.get("vec_w", f.top)
        ops.vec_gate_up(st.x, dim, logits, f.top, w.gate_up, w.shared_gate_up, f.ff, f.shared_ff, f.limit, f.shared_limit, GATE_ALPHA,
                        hidden, ids, sw)
        ops.vec_down(hidden, ids, sw, f.top, w.down, w.shared_down, f.ff, f.shared_ff, dim, y)
        st.pending = Pending(y, w.norm2)

    # -- a portion of tokens --
    def prefill(self, x: torch.Tensor, xh: torch.Tensor, rows: int, cur_pos: torch.Tensor) -> None:
        """x [portion, pad8(dim)] f32 residual, xh the same as activations; both are advanced."""
        m, w, sc, eps, dim, p, t = self.a.mixer, self.w, self.sc, self.args.eps, self.args.dim, self.portion, self.dtype
        qkv = sc.get("qkv", p, pad(self.n_q + self.n_kv))
        ops.gemm(xh, w.qkv, qkv, rows, self.n_q + self.n_kv, dim)
        q = sc.get("q", p, m.heads, pad(m.dim, 16), dtype=t)
        ops.qkv_rows(qkv, w.q_gain, w.k_gain, eps, self.v_mode, w.lam, self._v_first(p), rows, m, self.cache, cur_pos, q)
        att = sc.get("att", p, pad(m.heads * m.vdim), dtype=t)
        ops.attn_rows(q, m, self.cache, cur_pos, rows, att)
        y = sc.get("y", p, pad(dim))
        ops.gemm(att, w.o, y, rows, dim, m.heads * m.vdim)
        ops.residual_norm(x, xh, w.norm1, eps, dim, rows, y=y)
        f = self.a.mlp
        if f is None:
            return
        logits = sc.get("router", p, pad(f.experts))
        ops.gemm(xh, w.router, logits, rows, f.experts, dim, bias=w.router_bias)
        ids, rank, slot_row = (sc.get(n, p, f.top, dtype=I32) for n in ("ids", "rank", "slot_row"))
        sw, counts = sc.get("slot_w", p, f.top), sc.get("counts", f.experts, dtype=I32)
        ops.route_rows(logits, rows, f.experts, f.top, ids, sw, rank, counts)
        xs = sc.get("xs", p * f.top, pad(dim), dtype=t)
        ops.gather_rows(xh, rows, dim, f.experts, f.top, ids, rank, counts, xs, slot_row)
        hid = sc.get("hid", p * f.top, pad(f.ff), dtype=t)
        ops.gemm(xs, w.gate_up, hid, rows * f.top, f.ff, dim, gated=(f.limit, GATE_ALPHA), n_groups=f.experts, counts=counts)
        ye = sc.get("ye", p * f.top, pad(dim), dtype=t)
        ops.gemm(hid, w.down, ye, rows * f.top, dim, f.ff, n_groups=f.experts, counts=counts)
        ysh = None
        if f.shared_ff:
            hsh = sc.get("hsh", p, pad(f.shared_ff), dtype=t)
            ops.gemm(xh, w.shared_gate_up, hsh, rows, f.shared_ff, dim, gated=(f.shared_limit, GATE_ALPHA))
            ysh = sc.get("ysh", p, pad(dim), dtype=t)
            ops.gemm(hsh, w.shared_down, ysh, rows, dim, f.shared_ff)
        ops.residual_norm(x, xh, w.norm2, eps, dim, rows, experts=ye, slot_row=slot_row, slot_w=sw, shared=ysh)
