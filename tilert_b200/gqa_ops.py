"""Wrappers of the operators in ``include/tilert_gqa.h``: tensors in, raw pointers and the current CUDA stream out.
Outputs are caller-allocated.  The operators are mechanisms shared by any decoder that uses them (norms on an f32
residual, grouped products, windowed attention over a ring of cached rows, attention over a latent cache, routed experts);
a model decides sizes and order."""

from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

import tilert_b200 as _tb

_TYPE = "ralasun"  # the backend that carries these operators
BF16, F32, I32, I64 = torch.bfloat16, torch.float32, torch.int32, torch.int64
VMIX_NONE, VMIX_FIRST, VMIX_BLEND = 0, 1, 2


def pad(n: int, m: int = 8) -> int:
    return (n + m - 1) // m * m


@dataclass(frozen=True)
class Norm:
    """A norm's constants, f32 with zeros beyond the logical length; ``centered``: layer norm, else RMS norm."""

    gain: torch.Tensor
    bias: torch.Tensor | None = None
    centered: bool = False


def _norm(n) -> Norm:
    """A bare gain stands for an RMS norm without bias."""
    return n if isinstance(n, Norm) else Norm(n)


def _norms(first, second):
    """(gain, bias, gain2, bias2, centered) of two optional norms of one launch."""
    a, b = (None if n is None else _norm(n) for n in (first, second))
    kinds = {n.centered for n in (a, b) if n is not None}
    if len(kinds) > 1:
        raise ValueError("the norms of one launch are of one kind")
    return (*((None, None) if a is None else (_p(a.gain), _p(a.bias))), *((None, None) if b is None else (_p(b.gain), _p(b.bias))),
            int(kinds.pop()) if kinds else 0)


def _p(t: torch.Tensor | None):
    return None if t is None else t.data_ptr()


def _call(name: str, ref: torch.Tensor, *args) -> None:
    if not ref.is_cuda:
        raise ValueError(f"{name}: CUDA tensors are needed (there is no CPU path)")
    fn = getattr(_tb.lib(_TYPE), f"tilert_gqa_{name}_op")
    _tb.check(fn(_tb.tilert_init(ref.device.index, _TYPE), *args, torch.cuda.current_stream(ref.device).cuda_stream), _TYPE)


def _need(name: str, t: torch.Tensor | None, dtype, optional: bool = False) -> None:
    if t is None:
        if optional:
            return
        raise ValueError(f"{name} must be given")
    if t.dtype != dtype or t.stride(-1) != 1 and t.shape[-1] != 1:
        raise ValueError(f"{name} must be a {dtype} tensor with contiguous rows, got {t.dtype} strides {tuple(t.stride())}")


def _f32(*acts: torch.Tensor | None) -> int:
    """1 for the exact mode; every activation operand of a call has the same type."""
    kinds = {t.dtype for t in acts if t is not None}
    if kinds == {F32}:
        return 1
    if kinds == {BF16}:
        return 0
    raise ValueError(f"activations must all be bfloat16 or all be float32, got {kinds}")


def num_sms(device) -> int:
    return int(_tb.lib(_TYPE).tilert_gqa_num_sms(_tb.tilert_init(torch.device(device).index or 0, _TYPE)))


def head_blocks(heads: int, kv_heads: int) -> int:
    return int(_tb.lib(_TYPE).tilert_gqa_head_blocks(heads, kv_heads))


def embed_norm(tokens, table, gain, eps: float, dim: int, x, xh=None, *, exact: bool = False) -> None:
    """x[t] = rms(table[tokens[t]]) * gain (f32; ``gain`` None: the row as it is), also as activations in ``xh``."""
    _need("tokens", tokens, I64)
    _need("table", table, BF16)
    _need("x", x, F32)
    f32 = int(exact) if xh is None else _f32(xh)
    _call("embed_norm", x, _p(tokens), _p(table), table.stride(0), table.shape[0], _p(gain), eps, tokens.numel(), dim, _p(x),
          x.stride(-2), _p(xh), 0 if xh is None else xh.stride(-2), f32)


def residual_norm(x, xh, norm, eps: float, dim: int, rows: int, *, y=None, experts=None, slot_row=None, slot_w=None,
                  shared=None, add=None, norm2=None) -> None:
    """x += norm(y) (+ add), xh = x or norm2(x); y is given, or combined from expert output rows (+ the shared expert's), or
    there is none (``norm`` None).  ``xh`` None: x alone."""
    _need("x", x, F32)
    _need("y", y, F32, optional=True)
    gain, bias, gain2, bias2, centered = _norms(norm, norm2)
    acts = [t for t in (xh, experts, shared) if t is not None]
    _call("residual_norm", x, _p(y), 0 if y is None else y.stride(-2), _p(experts), 0 if experts is None else experts.stride(-2),
          _p(slot_row), _p(slot_w), 0 if slot_w is None else slot_w.shape[-1], _p(shared), 0 if shared is None else shared.stride(-2),
          gain, bias, _p(add), gain2, bias2, centered, eps, rows, dim, _p(x), x.stride(-2), _p(xh), 0 if xh is None else xh.stride(-2),
          _f32(*acts) if acts else 1)


def gather_norm(x, rows, norm, eps: float, dim: int, out) -> None:
    _need("x", x, F32)
    _need("rows", rows, I32)
    n = _norm(norm)
    _call("gather_norm", x, _p(x), x.stride(-2), _p(rows), rows.numel(), _p(n.gain), _p(n.bias), int(n.centered), eps, dim, _p(out),
          out.stride(-2), _f32(out))


def gemm(x, w, out, rows: int, n: int, k: int, *, gated: tuple[float, float] | None = None, n_groups: int = 0, counts=None,
         bias=None) -> None:
    """out[t, :n] = W x[t] (+ bias); ``gated`` = (limit, alpha) for a weight of n gate and n up rows; ``n_groups`` weights
    with ``counts`` rows each, or ``rows`` rows each without counts."""
    _need("w", w, BF16)
    f32 = _f32(x)
    limit, alpha = gated if gated is not None else (0.0, 0.0)
    if out.dtype != F32 and out.dtype != x.dtype:
        raise ValueError(f"gemm: output type {out.dtype} does not fit input type {x.dtype}")
    _call("gemm", x, _p(x), x.stride(-2), rows, _p(w), w.stride(-2), n, k, int(gated is not None), limit, alpha, n_groups, _p(counts),
          _p(bias), _p(out), out.stride(-2), int(out.dtype == F32), f32)


def qkv_rows(qkv, q_gain, k_gain, eps: float, v_mode: int, lam, v_first, rows: int, mix, cache, pos, q) -> None:
    """Normalise queries and keys, mix values, write the cache rows of positions *pos .. *pos + rows - 1."""
    _need("qkv", qkv, F32)
    _call("qkv_rows", q, _p(qkv), qkv.stride(-2), _p(q_gain), _p(k_gain), eps, v_mode, _p(lam), _p(v_first), rows, mix.heads, mix.kv_heads,
          mix.dim, mix.vdim, _p(pos), _p(q), _p(cache.k), _p(cache.v), cache.ring, _f32(q, cache.k, cache.v))


def attn_rows(q, mix, cache, pos, rows: int, out) -> None:
    _call("attn_rows", q, _p(q), _p(cache.k), _p(cache.v), rows, mix.heads, mix.kv_heads, mix.dim, mix.vdim, _p(pos), cache.window,
          cache.ring, mix.scale, _p(out), out.stride(-2), _f32(q, cache.k, cache.v, out))


def route_rows(logits, rows: int, n_experts: int, top: int, ids, w, rank, counts) -> None:
    _need("logits", logits, F32)
    _call("route_rows", logits, _p(logits), logits.stride(-2), rows, n_experts, top, _p(ids), _p(w), _p(rank), _p(counts))


def gather_rows(x, rows: int, dim: int, n_experts: int, top: int, ids, rank, counts, xs, slot_row) -> None:
    _call("gather_rows", x, _p(x), x.stride(-2), rows, dim, n_experts, top, _p(ids), _p(rank), _p(counts), _p(xs), _p(slot_row),
          _f32(x, xs))


def _stage(x, y, gain, add, gain2, eps: float, x_out):
    _need("x", x, F32)
    g, b, g2, b2, centered = _norms(gain, gain2)
    return _p(x), _p(y), g, b, _p(add), g2, b2, centered, eps, _p(x_out)


def vec_dense(x, w, out, n: int, k: int, *, y=None, gain=None, add=None, gain2=None, eps: float = 0.0, x_out=None, bias=None) -> None:
    """One-token product with the norm / residual step of its input fused in (see the header); ``gain`` and ``gain2`` are
    norms, or bare gains of RMS norms."""
    _need("w", w, BF16)
    _call("vec_dense", x, *_stage(x, y, gain, add, gain2, eps, x_out), _p(w), w.stride(-2), _p(bias), n, k, _p(out))


def vec_gated(x, w, out, n: int, k: int, limit: float, alpha: float, *, y=None, gain=None, add=None, gain2=None, eps: float = 0.0,
              x_out=None) -> None:
    """The same with the gated unit of a dense feed-forward, w [2, n, k]."""
    _need("w", w, BF16)
    _call("vec_gated", x, *_stage(x, y, gain, add, gain2, eps, x_out), _p(w), w.stride(-2), n, k, limit, alpha, _p(out))


def vec_attn(qkv, q_gain, k_gain, eps: float, v_mode: int, lam, v_first, mix, cache, pos, n_splits: int, part, counter, out) -> None:
    _need("qkv", qkv, F32)
    _call("vec_attn", qkv, _p(qkv), _p(q_gain), _p(k_gain), eps, v_mode, _p(lam), _p(v_first), mix.heads, mix.kv_heads, mix.dim, mix.vdim,
          _p(pos), cache.window, cache.ring, mix.scale, _p(cache.k), _p(cache.v), n_splits, _p(part), _p(counter), _p(out),
          _f32(cache.k, cache.v))


def vec_gate_up(x, dim: int, logits, top: int, w, w_sh, ff: int, ff_sh: int, limit: float, limit_sh: float, alpha: float, hidden,
                slot_ids, slot_w) -> None:
    _need("w", w, BF16)
    _call("vec_gate_up", x, _p(x), dim, _p(logits), w.shape[0], top, _p(w), _p(w_sh), w.stride(-2), ff, ff_sh, limit, limit_sh, alpha,
          _p(hidden), _p(slot_ids), _p(slot_w))


def vec_down(hidden, slot_ids, slot_w, top: int, w, w_sh, ff: int, ff_sh: int, dim: int, out) -> None:
    _call("vec_down", hidden, _p(hidden), _p(slot_ids), _p(slot_w), top, _p(w), _p(w_sh), ff, ff_sh, dim, _p(out))


# -- attention over a latent cache; ``mix`` has heads, dim, rot_dim, vdim, kv_rank, scale, ``rope`` is a Rotation --
@dataclass(frozen=True)
class Rotation:
    """table [positions, dims] f32: dims / 2 cosines, then dims / 2 sines per position."""

    table: torch.Tensor
    interleaved: bool

    def args(self):
        return _p(self.table), self.table.shape[0], self.table.shape[1], int(self.interleaved)


def rotation_table(base: float, dims: int, positions: int, device) -> torch.Tensor:
    """Angle of pair i at position p: p * base^(-2i / dims)."""
    f = torch.pow(torch.tensor(base, dtype=torch.float64), -torch.arange(0, dims, 2, dtype=torch.float64) / max(dims, 1))
    a = torch.arange(positions, dtype=torch.float64)[:, None] * f
    return torch.cat([torch.cos(a), torch.sin(a)], dim=1).to(device, F32).contiguous()


def latent_row_len(rank: int, rot: int) -> int:
    """Elements of a cache row: the latent padded to 16, the rotated part behind it, all padded to 32."""
    return pad(pad(rank, 16) + rot, 32)


def latent_blocks(mix, tokens: int, dtype) -> int:
    return int(_tb.lib(_TYPE).tilert_gqa_latent_blocks(mix.heads, tokens, mix.kv_rank, mix.rot_dim, int(dtype == F32)))


def expanded_fits(mix) -> bool:
    return bool(_tb.lib(_TYPE).tilert_gqa_expanded_fits(mix.dim, mix.rot_dim, mix.vdim))


def latent_tokens(z, off_c: int, off_r: int, q_rank: int, q_gain, c_gain, eps: float, rows: int, mix, rope: Rotation, cache, pos, cq) -> None:
    """Query latents normed into ``cq``, the cache rows of positions *pos .. *pos + rows - 1."""
    _need("z", z, F32)
    _call("latent_tokens", z, _p(z), z.stride(-2), q_rank, off_c, off_r, _p(q_gain), _p(c_gain), eps, rows, mix.kv_rank, mix.rot_dim,
          *rope.args(), _p(pos), cache.ring, _p(cq), cq.stride(-2), _p(cache.rows), _f32(cq, cache.rows))


def latent_queries(q, rows: int, mix, rope: Rotation, pos, out, lat=None) -> None:
    _need("q", q, F32)
    _need("lat", lat, F32, optional=True)
    _call("latent_queries", q, _p(q), q.stride(-2), rows, mix.heads, mix.dim, mix.rot_dim, *rope.args(), _p(pos), _p(out), _p(lat),
          mix.kv_rank, _f32(out))


def latent_attn(lat, cache, tokens: int, mix, pos, n_splits: int, part) -> None:
    _need("lat", lat, F32)
    need = mix.heads * tokens * n_splits * (pad(mix.kv_rank, 16) + 2)
    if part.numel() < need:
        raise ValueError(f"part holds {part.numel()} elements, {need} are needed")
    _call("latent_attn", lat, _p(lat), _p(cache.rows), tokens, mix.heads, mix.kv_rank, mix.rot_dim, _p(pos), cache.window, cache.ring,
          mix.scale, n_splits, _p(part), _f32(cache.rows))


def latent_merge(part, tokens: int, mix, n_splits: int, sink, out) -> None:
    _call("latent_merge", part, _p(part), tokens, mix.heads, n_splits, mix.kv_rank, mix.rot_dim, _p(sink), _p(out), out.stride(-2), _f32(out))


def gate_heads(o, rows: int, heads: int, vdim: int, gate, per_head: bool, out) -> None:
    _need("o", o, F32)
    _call("gate_heads", o, _p(o), o.stride(-2), rows, heads, vdim, _p(gate), 0 if gate is None else gate.stride(-2), int(per_head), _p(out),
          out.stride(-2), _f32(out))


def expanded_attn(q, kv, cache, rows: int, mix, pos, sink, gate, per_head: bool, out) -> None:
    for t in (q, kv, cache.rows, out):
        _need("operand", t, BF16)
    _call("expanded_attn", q, _p(q), _p(kv), _p(cache.rows), rows, mix.heads, mix.dim, mix.rot_dim, mix.vdim, mix.kv_rank, _p(pos),
          cache.window, cache.ring, mix.scale, _p(sink), _p(gate), 0 if gate is None else gate.stride(-2), int(per_head), _p(out),
          out.stride(-2))


def vec_absorb(q, w, mix, rope: Rotation, c, kr, c_gain, eps: float, pos, cache, lat) -> None:
    """One token: absorbed, rotated queries into ``lat`` [heads, row], and its cache row."""
    _need("w", w, BF16)
    _call("vec_absorb", q, _p(q), mix.heads, mix.dim, mix.kv_rank, mix.rot_dim, _p(w), w.stride(-2), *rope.args(), _p(c), _p(kr), _p(c_gain),
          eps, _p(pos), cache.ring, _p(lat), _p(cache.rows), _f32(cache.rows))


def vec_value(part, w, mix, n_splits: int, sink, gate, per_head: bool, out) -> None:
    """One token: merged parts through the value expansion, gated, [heads * vdim]."""
    _need("w", w, BF16)
    _call("vec_value", part, _p(part), mix.heads, mix.vdim, mix.kv_rank, mix.rot_dim, n_splits, _p(sink), _p(w), w.stride(-2), _p(gate),
          int(per_head), _p(out))


def sample(logits, config, token_out, *, seed=0, step=None, step_value=0, token_logprob=None, topn_logprobs=None,
           topn_indices=None) -> None:
    """Same operator as ``models.deepseek_v3_2.ops.sample``, from this backend's library."""
    _need("logits", logits, F32)
    _need("token_out", token_out, I32)
    rows = logits.numel() // logits.shape[-1]
    _call("sample", logits, _p(logits), logits.shape[-1], rows, logits.shape[-1], _p(config), seed & ((1 << 63) - 1), _p(step), step_value,
          _p(token_out), _p(token_logprob), _p(topn_logprobs), _p(topn_indices))
