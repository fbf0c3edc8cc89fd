"""Weights, caches and the operator sequence of one Rozesun layer.

A layer norms the input and the output of its sublayers: x += n1b(attention(n1(x))), x += n2b(ff(n2(x))).  Attention goes
through latents: the queries' own, and one of keys and values, which (with a rotated key part shared by the heads) is all
that is cached.  Three forms of it:

* ``decode`` -- one token, f32 vectors, eight launches per layer: the products of the normed input (both latents, key part,
  gate), queries, key expansion moved onto the queries + rotation + cache row, attention over the latent rows, merge +
  value expansion + gate, output product, gate/up, down.  What lies between two sublayers rides on the next launch's
  input staging (``Stream``).
* ``prefill``, absorbed -- the same algebra for a portion of tokens (few tokens, or the exact f32 mode).
* ``prefill``, expanded -- keys and values of the cache rows in use are expanded first: more work per key, less per query
  and key, for portions of many tokens.
"""

from __future__ import annotations

import torch

from tilert_b200 import gqa_ops as ops
from tilert_b200.gqa_ops import BF16, F32, pad
from tilert_b200.kv_cache import LatentCache

from ..blocks import Pending, RowStream, Scratch, Stream, layer_norm, padded_rows, padded_vec
from .model_args import GATE_ALPHA, LayerArgs, MixerArgs, RozesunArgs


def _row_blocks(*parts: torch.Tensor) -> torch.Tensor:
    """The parts' rows below each other, each part filled with zero rows to a multiple of eight."""
    return torch.cat([torch.nn.functional.pad(p, (0, 0, 0, pad(p.shape[0]) - p.shape[0])) for p in parts])


def _head_rows(w: torch.Tensor, heads: int, m: int) -> torch.Tensor:
    """[heads * n, k] -> [heads, n filled with zero rows to a multiple of m, k]."""
    w = w.reshape(heads, -1, w.shape[-1])
    return torch.nn.functional.pad(w, (0, 0, 0, pad(w.shape[1], m) - w.shape[1]))


class LayerWeights:
    """One layer's tensors, read under their checkpoint names from ``sd`` (any key -> tensor mapping)."""

    def __init__(self, args: RozesunArgs, sd, li: int, device, expanded: bool):
        """``expanded``: the weights of the expanded form too."""
        a = args.layers[li]
        m, f, dev = a.mixer, a.mlp, torch.device(device)
        mix, mlp = f"l{li}.mix", f"l{li}.mlp"
        h, r = m.heads, m.kv_rank
        want = {"dq": (m.q_rank, args.dim), "dq.norm": (m.q_rank,), "uq": (h * (m.dim + m.rot_dim), m.q_rank), "dkv": (r + m.rot_dim, args.dim),
                "dkv.norm": (r,), "uk": (h * m.dim, r), "uv": (h * m.vdim, r), "g": (m.gate_rows, args.dim), "o": (args.dim, h * m.vdim)}
        if m.sink:
            want["sink"] = (h,)
        t = {n: sd[f"{mix}.{n}"].to(dev) for n in want}
        if f is not None:
            want |= {"gate": (f.ff, args.dim), "up": (f.ff, args.dim), "down": (args.dim, f.ff)}
            t |= {n: sd[f"{mlp}.{n}"].to(dev) for n in ("gate", "up", "down")}
        for n, shape in want.items():
            if tuple(t[n].shape) != shape:
                raise ValueError(f"layer {li}: {n} has shape {tuple(t[n].shape)}, the configuration says {shape}")

        # everything that reads the layer's normed input, one product: [query latent | latent | key part | gate]
        self.off_c = pad(m.q_rank)
        self.off_r = self.off_c + pad(r)
        self.off_g = self.off_r + pad(m.rot_dim)
        self.z = padded_rows(_row_blocks(t["dq"], t["dkv"][:r], t["dkv"][r:], t["g"]), dev)
        self.q_gain, self.c_gain = padded_vec(t["dq.norm"], dev), padded_vec(t["dkv.norm"], dev)
        # per head [unrotated, zero rows | rotated, zero rows]
        uq = t["uq"].view(h, m.dim + m.rot_dim, m.q_rank)
        self.uq = padded_rows(torch.cat([_head_rows(p.reshape(-1, m.q_rank), h, 8) for p in (uq[:, : m.dim], uq[:, m.dim:])], dim=1)
                              .flatten(0, 1), dev)
        self.uk_t = padded_rows(t["uk"].view(h, m.dim, r).transpose(1, 2), dev)            # [heads, rank, pad8(dim)]
        self.kv = None
        if expanded:  # keys of all heads, then values, in rows of 16
            self.kv = padded_rows(torch.cat([_head_rows(t[n], h, 16).flatten(0, 1) for n in ("uk", "uv")]), dev)
        if expanded and m.vdim % 16 == 0:
            self.uv = self.kv[h * pad(m.dim, 16):].view(h, m.vdim, -1)                    # [heads, vdim, pad8(rank)]
        else:
            self.uv = padded_rows(t["uv"].view(h, m.vdim, r), dev)
        self.sink = t["sink"].to(F32).contiguous() if m.sink else None
        self.o = padded_rows(t["o"], dev)
        self.norm1, self.norm1b = (layer_norm(sd, f"l{li}.{n}", dev) for n in ("norm1", "norm1b"))
        self.norm2 = self.norm2b = self.gate_up = self.down = None
        if f is not None:
            self.norm2, self.norm2b = (layer_norm(sd, f"l{li}.{n}", dev) for n in ("norm2", "norm2b"))
            self.gate_up = padded_rows(torch.stack([t["gate"], t["up"]]), dev)
            self.down = padded_rows(t["down"], dev)

    def weight_bytes(self) -> int:
        """Bytes of weights one decode step streams from HBM."""
        ts = [self.z, self.uq, self.uk_t, self.uv, self.o] + ([self.gate_up, self.down] if self.down is not None else [])
        return 2 * sum(t.numel() for t in ts)


def expansion_pays(m: MixerArgs, rows: int, visible: int, cached: int) -> bool:
    """Whether expanding the keys and values of ``cached`` rows costs a portion of ``rows`` tokens, that see ``visible``
    keys each, fewer products than working on the latents."""
    absorbed = rows * (visible * (2 * m.kv_rank + m.rot_dim) + m.kv_rank * (m.dim + m.vdim))
    expanded = rows * visible * (m.dim + m.rot_dim + m.vdim) + cached * m.kv_rank * (m.dim + m.vdim)
    return expanded < absorbed


class RozesunLayer:
    def __init__(self, args: RozesunArgs, li: int, weights: LayerWeights, rope: ops.Rotation, scratch: Scratch, portion: int, dtype,
                 device, passes: int):
        self.args, self.a, self.w, self.rope, self.sc = args, args.layers[li], weights, rope, scratch
        self.dtype, self.portion = dtype, portion
        m = self.a.mixer
        self.caches = [LatentCache(m.kv_rank, m.rot_dim, m.window, args.max_seq_len, portion, device, dtype) for _ in range(passes)]
        self.sms = ops.num_sms(device)
        self.z_len = weights.off_g + m.gate_rows
        self.ldh = pad(m.dim) + pad(m.rot_dim)

    def _splits(self, tokens: int, keys: int) -> int:
        """Parts of the key range, of ``per`` tiles of 64 keys each: no more than fill the SMs, and no more than pay (a tile
        takes about as long as the merge of 24 parts)."""
        tiles = (keys + 63) // 64
        least = -(-tiles // max(1, self.sms // ops.latent_blocks(self.a.mixer, tokens, self.dtype)))
        return min((-(-tiles // per) for per in range(least, least + 4)), key=lambda n: 24 * -(-tiles // n) + n)

    # -- one token --
    def decode(self, st: Stream, nr: int, cur_pos: torch.Tensor, length: int) -> None:
        """Pass ``nr``; ``length``: an upper bound of the sequence's length including this token."""
        m, w, sc, eps, dim, cache = self.a.mixer, self.w, self.sc, self.args.eps, self.args.dim, self.caches[nr]
        z = sc.get("vec_z", pad(self.z_len))
        st.dense(w.z, z, self.z_len, dim, eps, gain2=w.norm1)
        q = sc.get("vec_q", m.heads * self.ldh)
        ops.vec_dense(z, w.uq, q, m.heads * self.ldh, m.q_rank, gain2=w.q_gain, eps=eps)
        lat = sc.get("vec_lat", m.heads, cache.rows.shape[1])
        ops.vec_absorb(q, w.uk_t, m, self.rope, z[w.off_c:], z[w.off_r:], w.c_gain, eps, cur_pos, cache, lat)
        n_splits = self._splits(1, cache.visible(length))
        part = sc.get("vec_part", m.heads * n_splits * (pad(m.kv_rank, 16) + 2))
        ops.latent_attn(lat, cache, 1, m, cur_pos, n_splits, part)
        att = sc.get("vec_att", pad(m.heads * m.vdim))
        ops.vec_value(part, w.uv, m, n_splits, w.sink, z[w.off_g:], m.gate_per_head, att)
        y = sc.get("vec_y", pad(dim))
        ops.vec_dense(att, w.o, y, dim, m.heads * m.vdim)
        st.pending = Pending(y, w.norm1b)
        f = self.a.mlp
        if f is None:
            return
        hidden = sc.get("vec_hidden", pad(f.ff))
        st.gated(w.gate_up, hidden, f.ff, dim, f.limit, GATE_ALPHA, eps, gain2=w.norm2)
        ops.vec_dense(hidden, w.down, y, dim, f.ff)
        st.pending = Pending(y, w.norm2b)

    # -- a portion of tokens --
    def prefill(self, st: RowStream, nr: int, cur_pos: torch.Tensor, pos: int) -> None:
        """Pass ``nr``; ``pos``: the position of the first row, as ``cur_pos`` holds it."""
        m, w, sc, eps, dim, t, n = self.a.mixer, self.w, self.sc, self.args.eps, self.args.dim, self.dtype, st.rows
        cache = self.caches[nr]
        h = st.normed(w.norm1)
        z = sc.flat("z", n, pad(self.z_len))
        ops.gemm(h, w.z, z, n, self.z_len, dim)
        cq = sc.get("cq", self.portion, pad(m.q_rank), dtype=t)
        ops.latent_tokens(z, w.off_c, w.off_r, m.q_rank, w.q_gain, w.c_gain, eps, n, m, self.rope, cache, cur_pos, cq)
        q = sc.flat("q", n, m.heads * self.ldh)
        ops.gemm(cq, w.uq, q, n, m.heads * self.ldh, m.q_rank)
        att = sc.get("att", self.portion, pad(m.heads * m.vdim), dtype=t)
        length = pos + n
        cached = min(length, cache.ring)
        if w.kv is not None and expansion_pays(m, n, min(length, cache.window or length), cached):
            self._expanded(q, z, n, cache, cur_pos, cached, att)
        else:
            self._absorbed(q, z, n, cache, cur_pos, length, att)
        y = sc.get("y", self.portion, pad(dim))
        ops.gemm(att, w.o, y, n, dim, m.heads * m.vdim)
        st.pending = Pending(y, w.norm1b)
        f = self.a.mlp
        if f is None:
            return
        hid = sc.get("hid", self.portion, pad(f.ff), dtype=t)
        ops.gemm(st.normed(w.norm2), w.gate_up, hid, n, f.ff, dim, gated=(f.limit, GATE_ALPHA))
        ops.gemm(hid, w.down, y, n, dim, f.ff)
        st.pending = Pending(y, w.norm2b)

    def _expanded(self, q, z, n: int, cache: LatentCache, cur_pos, cached: int, att) -> None:
        m, w, sc = self.a.mixer, self.w, self.sc
        wide = pad(m.dim, 16) + pad(m.rot_dim, 16)
        qe = sc.flat("qe", n, m.heads, wide, dtype=self.dtype)
        ops.latent_queries(q, n, m, self.rope, cur_pos, qe)
        kv = sc.flat("kv", cached, w.kv.shape[0], dtype=self.dtype)
        ops.gemm(cache.rows, w.kv, kv, cached, w.kv.shape[0], m.kv_rank)
        ops.expanded_attn(qe, kv, cache, n, m, cur_pos, w.sink, z[:, w.off_g:], m.gate_per_head, att)

    def _absorbed(self, q, z, n: int, cache: LatentCache, cur_pos, length: int, att) -> None:
        m, w, sc, t = self.a.mixer, self.w, self.sc, self.dtype
        rank, hn = m.kv_rank, m.heads * n
        qn = sc.flat("qn", hn, pad(m.dim), dtype=t)
        lat = sc.flat("lat", hn, cache.rows.shape[1])
        ops.latent_queries(q, n, m, self.rope, cur_pos, qn, lat)
        ops.gemm(qn, w.uk_t, lat, n, rank, m.dim, n_groups=m.heads)
        n_splits = self._splits(n, cache.visible(length, n))
        part = sc.flat("part", hn * n_splits * (pad(rank, 16) + 2))
        ops.latent_attn(lat, cache, n, m, cur_pos, n_splits, part)
        c = sc.flat("c", hn, pad(rank), dtype=t)
        ops.latent_merge(part, n, m, n_splits, w.sink, c)
        o = sc.flat("o", hn, pad(m.vdim))
        ops.gemm(c, w.uv, o, n, m.vdim, rank, n_groups=m.heads)
        ops.gate_heads(o, n, m.heads, m.vdim, z[:, w.off_g:], m.gate_per_head, att)

    def weight_bytes(self) -> int:
        return self.w.weight_bytes() * len(self.caches)
