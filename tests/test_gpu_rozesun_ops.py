"""The mechanisms that the Rozesun design adds to ``include/tilert_gqa.h``, one by one against the plain restatement in
``oracle/rozesun.py``, in both activation types, at sizes that are not multiples of anything convenient."""

import pytest
import torch

from oracle import ralasun as RR
from oracle import rozesun as R

pytestmark = pytest.mark.gpu

BF16, F32, F64, I32, I64 = torch.bfloat16, torch.float32, torch.float64, torch.int32, torch.int64
TYPES = [F32, BF16]
ALPHA = 1.702


@pytest.fixture(scope="module")
def ops():
    import tilert_b200 as tb
    from tilert_b200 import gqa_ops

    tb.load_backend("ralasun")
    tb.tilert_init(0, "ralasun")
    yield gqa_ops
    assert tb.device_status(0, "ralasun") == 0


def rnd(seed, *shape, std=1.0, mean=0.0, dtype=F32):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * std + mean).to(dtype)


def padded(t, m=8):
    k = t.shape[-1]
    return torch.nn.functional.pad(t, (0, (k + m - 1) // m * m - k)).contiguous().cuda()


def close(name, ref, out, dtype, exact=2e-6, half=6e-3):
    ref, out = ref.double().cpu(), out.double().cpu()
    assert ref.shape == out.shape, (name, ref.shape, out.shape)
    err = ((ref - out).pow(2).mean().sqrt() / ref.pow(2).mean().sqrt().clamp_min(1e-30)).item()
    worst = ((ref - out).abs().max() / ref.abs().max().clamp_min(1e-30)).item()
    lim = exact if dtype == F32 else half
    assert err <= lim and worst <= 8 * lim, f"{name}: rms {err:.2e}, worst {worst:.2e}, limit {lim:.0e}"


class LN:
    """Constants of a layer norm, and the norm itself in f64."""

    def __init__(self, ops, seed, dim, eps):
        self.w, self.b, self.eps = rnd(seed, dim, std=0.3, mean=1.0), rnd(seed + 1, dim, std=0.5), eps
        self.dev = ops.Norm(padded(self.w), padded(self.b), centered=True)

    def __call__(self, x):
        return R.layer_norm(x.double(), self.w.double(), self.b.double(), self.eps)


# ------------------------------------------------------------------ norms
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("dim", [50, 256, 1030])
def test_layer_norms_on_the_residual(ops, dtype, dim):
    rows, eps = 9, 1e-2
    n1, n2 = LN(ops, 10, dim, eps), LN(ops, 20, dim, eps)
    # (a mean far from zero: the deviations must not come from a difference of squares)
    x0, y, add = rnd(0, rows, dim), rnd(1, rows, dim, std=0.7, mean=40.0), rnd(2, dim)
    for with_y, with_add, with_norm in ((1, 0, 1), (1, 1, 1), (0, 1, 1), (1, 1, 0), (0, 0, 1)):
        x, xh = padded(x0), torch.zeros(rows, ops.pad(dim), dtype=dtype, device="cuda")
        ops.residual_norm(x, xh if with_norm else None, n1.dev if with_y else None, eps, dim, rows, y=padded(y) if with_y else None,
                          add=padded(add) if with_add else None, norm2=n2.dev if with_norm else None)
        v = x0.double() + (n1(y) if with_y else 0) + (add.double() if with_add else 0)
        close("x", v, x[:, :dim], F32, exact=5e-6)
        if with_norm:
            close("xh", n2(v), xh[:, :dim], dtype, exact=5e-6)
    pick = torch.tensor([7, 0, 7], dtype=I32, device="cuda")
    out = torch.zeros(3, ops.pad(dim), dtype=dtype, device="cuda")
    ops.gather_norm(padded(y), pick, n2.dev, eps, dim, out)
    close("gathered", n2(y[[7, 0, 7]]), out[:, :dim], dtype, exact=5e-6)
    with pytest.raises(ValueError):  # one launch, one kind of norm
        ops.residual_norm(padded(x0), xh, n1.dev, eps, dim, rows, y=padded(y), norm2=padded(n2.w))


def test_plain_embedding(ops):
    table, toks = rnd(0, 37, 50, std=3.0, dtype=BF16), torch.tensor([5, 36, 0, 5])
    x = torch.zeros(4, 56, device="cuda")
    ops.embed_norm(toks.cuda(), padded(table), None, 1e-3, 50, x)
    assert torch.equal(x[:, :50].cpu(), table[toks].float())


@pytest.mark.parametrize("n,k", [(1, 8), (5, 30), (150, 201), (777, 4096), (300, 9001)])
def test_one_token_products_with_layer_norms(ops, n, k):
    eps = 1e-3
    n1, n2 = LN(ops, 10, k, eps), LN(ops, 20, k, eps)
    x, y, add = rnd(0, k), rnd(1, k, std=0.5, mean=9.0), rnd(2, k)
    w, g, u = (rnd(s, n, k, std=2 * k ** -0.5, dtype=BF16) for s in (3, 4, 5))
    wd, gu, out, xo = padded(w), padded(torch.stack([g, u])), torch.zeros(n, device="cuda"), torch.zeros(ops.pad(k), device="cuda")
    for kw, v in ((dict(y=padded(y), gain=n1.dev), x.double() + n1(y)),
                  (dict(y=padded(y), gain=n1.dev, add=padded(add)), x.double() + n1(y) + add.double()),
                  (dict(add=padded(add)), x.double() + add.double()), ({}, x.double())):
        for norm in (None, n2):
            h = v if norm is None else norm(v)
            ops.vec_dense(padded(x), wd, out, n, k, eps=eps, x_out=xo, gain2=None if norm is None else norm.dev, **kw)
            close("vector", v, xo[:k], F32, exact=5e-6)
            close("dense", w.double() @ h, out, F32, exact=1e-5)
            assert float(xo[k:].abs().sum()) == 0
            ops.vec_gated(padded(x), gu, out, n, k, 0.9, ALPHA, eps=eps, gain2=None if norm is None else norm.dev, **kw)
            close("gated", RR.gated_unit(g.double() @ h, u.double() @ h, 0.9), out, F32, exact=1e-5)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("rows", [1, 7, 70, 200])
def test_groups_of_equal_size(ops, dtype, rows):
    n, k, e = 45, 37, 5
    x, w = rnd(0, e, rows, k, dtype=dtype), rnd(1, e, n, k, std=k ** -0.5, dtype=BF16)
    out = torch.full((e * rows, n + 3), 7.0, device="cuda")
    ops.gemm(padded(x).flatten(0, 1), padded(w), out, rows, n, k, n_groups=e)
    close("groups", torch.einsum("erk,enk->ern", x.double(), w.double()).flatten(0, 1), out[:, :n], F32, exact=3e-6)
    assert bool((out[:, n:] == 7.0).all())


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("per_head", [True, False])
def test_output_gate(ops, dtype, per_head):
    rows, heads, vdim = 6, 5, 11
    o, z = rnd(0, heads, rows, vdim), rnd(1, rows, heads if per_head else heads * vdim, std=3.0)
    z[0, 0], z[0, 1] = 200.0, -200.0
    out = torch.zeros(rows, 56, dtype=dtype, device="cuda")
    ops.gate_heads(padded(o, 16), rows, heads, vdim, padded(z), per_head, out)
    close("gate", R.gate(o.transpose(0, 1).double(), z.double()), out[:, :55], dtype)
    ops.gate_heads(padded(o, 16), rows, heads, vdim, None, per_head, out)
    close("no gate", o.transpose(0, 1).flatten(1), out[:, :55], dtype)


# ------------------------------------------------------------------ attention over a latent cache
NEAR, WIDE = "latent_attention_2", "latent_attention"


class Latent:
    """One mixer without its outer products: what they would deliver is random, the weights in between are random; the
    plain result, and the launch forms over one cache."""

    def __init__(self, ops, mix, dtype, t, portion, seed=0, spike=None, sink=1.5):
        from tilert_b200.kv_cache import LatentCache
        from tilert_b200.models.rozesun.layer import LayerWeights
        from tilert_b200.models.rozesun.model_args import LayerArgs, RozesunArgs

        self.ops, self.m, self.dtype, self.eps, self.t, m = ops, mix, dtype, 1e-4, t, mix
        sizes = (m.q_rank, m.kv_rank, m.rot_dim, m.gate_rows)
        width = sum(sizes)
        pick = torch.eye(width, dtype=BF16).split(sizes)  # the mixer's input is what the projections would deliver, side by side
        h, (zq, zc, zr, zg) = (x := rnd(seed, t, width)), x.split(sizes, dim=1)
        uq, uk, uv = (rnd(seed + s, n, k, std=k ** -0.5, dtype=BF16) for s, n, k in
                      ((1, m.heads * (m.dim + m.rot_dim), m.q_rank), (2, m.heads * m.dim, m.kv_rank), (3, m.heads * m.vdim, m.kv_rank)))
        if spike is not None:  # all heads alike; key j lies along the absorbed query i
            i, j = spike
            uq, uk = uq[: m.dim + m.rot_dim].repeat(m.heads, 1), uk[: m.dim].repeat(m.heads, 1)
            uq[:, :] *= 4
            zc[j] = (uk[: m.dim].double().T @ (uq[: m.dim].double() @ RR.rms(zq[i].double(), self.eps))).float()
        w = {"l0.mix.dq": pick[0], "l0.mix.dkv": torch.cat(pick[1:3]), "l0.mix.g": pick[3], "l0.mix.uq": uq, "l0.mix.uk": uk, "l0.mix.uv": uv,
             "l0.mix.dq.norm": rnd(seed + 4, m.q_rank, std=0.2, mean=1.5).to(BF16), "l0.mix.dkv.norm": rnd(seed + 5, m.kv_rank, std=0.2, mean=1.2).to(BF16),
             "l0.mix.sink": rnd(seed + 6, m.heads, mean=sink).to(BF16), "l0.mix.o": torch.zeros(width, m.heads * m.vdim, dtype=BF16)}
        for n in ("norm1", "norm1b"):
            w |= {f"l0.{n}": torch.ones(width), f"l0.{n}.b": torch.zeros(width)}
        args = RozesunArgs(8, width, self.eps, 1.0, (LayerArgs(m, None),))
        self.w = LayerWeights(args, w, 0, "cuda", expanded=ops.expanded_fits(m))
        z = torch.zeros(t, ops.pad(self.w.off_g + m.gate_rows))
        for off, part in ((0, zq), (self.w.off_c, zc), (self.w.off_r, zr), (self.w.off_g, zg)):
            z[:, off: off + part.shape[1]] = part
        self.z = z.cuda()
        self.h, self.w64 = h.double(), {k: v.double() for k, v in w.items()}
        self.mixcfg = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "scale": m.scale,
                       "rot": {"base": m.rot_base, "dims": m.rot_dim}, "mask": {"size": m.window}}
        self.ref = self.plain()
        self.cache = LatentCache(m.kv_rank, m.rot_dim, m.window, t + 8, portion, "cuda", dtype)
        # what an earlier sequence left behind must not be seen
        rankp = ops.pad(m.kv_rank, 16)
        self.cache.rows[:, : m.kv_rank] = rnd(seed + 7, self.cache.ring, m.kv_rank, std=9.0).to("cuda", dtype)
        self.cache.rows[:, rankp: rankp + m.rot_dim] = rnd(seed + 8, self.cache.ring, m.rot_dim, std=9.0).to("cuda", dtype)
        self.rope = ops.Rotation(ops.rotation_table(m.rot_base, m.rot_dim, t + 8, "cuda"), m.interleaved)
        self.pos = torch.zeros(1, dtype=I32, device="cuda")
        self.ldh = ops.pad(m.dim) + ops.pad(m.rot_dim)

    def plain(self, window_off=0, without=None):
        """The restatement up to the gated heads [t, heads * vdim]; with a window of another size, or with the position
        ``without`` leaving a copy of the next one's key."""
        m, k, w, p = self.mixcfg, R.KINDS[self.m.kind], self.w64, "l0.mix"
        c, kr = R.latent_keys(self.h, w, p, m, self.eps, k["interleaved"])
        if without is not None:
            c[without] = c[without + 1]
        qn, qr = R.latent_queries(self.h, w, p, m, self.eps, k["interleaved"])
        o = R.latent_attend(qn, qr, c, kr, w[f"{p}.uk"], w[f"{p}.uv"], m["scale"], self.m.window + window_off if k["window"] else None,
                            w[f"{p}.sink"] if k["sink"] else None)
        return R.gate(o, self.h @ w[f"{p}.g"].T)

    def rows(self, lo, hi, form="absorbed", n_splits=1):
        """Positions lo .. hi - 1 as a portion."""
        ops, m, w, n, t = self.ops, self.m, self.w, hi - lo, self.dtype
        self.pos.fill_(lo)
        z = self.z[lo:hi].contiguous()
        cq = torch.zeros(n, ops.pad(m.q_rank), dtype=t, device="cuda")
        ops.latent_tokens(z, w.off_c, w.off_r, m.q_rank, w.q_gain, w.c_gain, self.eps, n, m, self.rope, self.cache, self.pos, cq)
        q = torch.zeros(n, m.heads * self.ldh, device="cuda")
        ops.gemm(cq, w.uq, q, n, m.heads * self.ldh, m.q_rank)
        att = torch.zeros(n, ops.pad(m.heads * m.vdim), dtype=t, device="cuda")
        if form == "expanded":
            qe = torch.zeros(n, m.heads, ops.pad(m.dim, 16) + ops.pad(m.rot_dim, 16), dtype=t, device="cuda")
            ops.latent_queries(q, n, m, self.rope, self.pos, qe)
            cached = min(hi, self.cache.ring)
            kv = torch.zeros(cached, w.kv.shape[0], dtype=t, device="cuda")
            ops.gemm(self.cache.rows, w.kv, kv, cached, w.kv.shape[0], m.kv_rank)
            ops.expanded_attn(qe, kv, self.cache, n, m, self.pos, w.sink, z[:, w.off_g:], m.gate_per_head, att)
        else:
            qn, lat = torch.zeros(m.heads * n, ops.pad(m.dim), dtype=t, device="cuda"), torch.zeros(m.heads * n, self.cache.rows.shape[1], device="cuda")
            ops.latent_queries(q, n, m, self.rope, self.pos, qn, lat)
            ops.gemm(qn, w.uk_t, lat, n, m.kv_rank, m.dim, n_groups=m.heads)
            part = torch.full((m.heads * n * n_splits * (ops.pad(m.kv_rank, 16) + 2),), float("nan"), device="cuda")  # empty parts stay unread
            ops.latent_attn(lat, self.cache, n, m, self.pos, n_splits, part)
            c, o = torch.zeros(m.heads * n, ops.pad(m.kv_rank), dtype=t, device="cuda"), torch.zeros(m.heads * n, ops.pad(m.vdim), device="cuda")
            ops.latent_merge(part, n, m, n_splits, w.sink, c)
            ops.gemm(c, w.uv, o, n, m.vdim, m.kv_rank, n_groups=m.heads)
            ops.gate_heads(o, n, m.heads, m.vdim, z[:, w.off_g:], m.gate_per_head, att)
        return att[:, : m.heads * m.vdim]

    def one(self, i, n_splits=1):
        """Position i by the one-token launches."""
        ops, m, w = self.ops, self.m, self.w
        self.pos.fill_(i)
        z = self.z[i].contiguous()
        q = torch.zeros(m.heads * self.ldh, device="cuda")
        ops.vec_dense(z, w.uq, q, m.heads * self.ldh, m.q_rank, gain2=w.q_gain, eps=self.eps)
        lat = torch.zeros(m.heads, self.cache.rows.shape[1], device="cuda")
        ops.vec_absorb(q, w.uk_t, m, self.rope, z[w.off_c:], z[w.off_r:], w.c_gain, self.eps, self.pos, self.cache, lat)
        part = torch.full((m.heads * n_splits * (ops.pad(m.kv_rank, 16) + 2),), float("nan"), device="cuda")
        ops.latent_attn(lat, self.cache, 1, m, self.pos, n_splits, part)
        att = torch.zeros(m.heads * m.vdim, device="cuda")
        ops.vec_value(part, w.uv, m, n_splits, w.sink, z[w.off_g:], m.gate_per_head, att)
        return att


def mixer(kind, heads, dim, rot, vdim, q_rank, kv_rank, window=None, scale=None, base=200.0):
    from tilert_b200.models.rozesun.model_args import MixerArgs

    return MixerArgs(kind, heads, dim, rot, vdim, q_rank, kv_rank, scale or (dim + rot) ** -0.5, base, window)


SHAPES = [(WIDE, 4, 32, 16, 24, 40, 48), (NEAR, 6, 40, 24, 24, 33, 65, 20), (NEAR, 5, 17, 6, 9, 21, 7, 64), (WIDE, 20, 64, 64, 136, 96, 272),
          (NEAR, 17, 24, 2, 8, 16, 130, 7), (WIDE, 2, 128, 64, 128, 200, 512), (NEAR, 1, 8, 8, 8, 8, 8, 1), (NEAR, 3, 200, 60, 250, 64, 640, 33)]


def forms(ops, mix, dtype):
    return ["absorbed"] + (["expanded"] if dtype == BF16 and ops.expanded_fits(mix) else [])


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("shape", SHAPES)
def test_attention_in_portions_and_token_by_token(ops, dtype, shape):
    mix, t = mixer(*shape), 150
    for form in forms(ops, mix, dtype):
        a = Latent(ops, mix, dtype, t, portion=70)
        lo = 0
        for n, s in ((64, 1), (2, 3), (70, 2), (3, 9)):
            close(f"{form} portion at {lo}", a.ref[lo: lo + n], a.rows(lo, lo + n, form, s), dtype, exact=5e-6, half=1.5e-2)
            lo += n
        for i, s in zip(range(lo, t), (1, 2, 5, 1, 3, 40, 1, 2, 4, 148, 8)):
            close(f"token {i}, {s} parts", a.ref[i], a.one(i, s), dtype, exact=5e-6, half=1.5e-2)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("kind", [WIDE, NEAR])
def test_decoding_past_many_turns_of_the_ring(ops, dtype, kind):
    mix, t = mixer(kind, 4, 32, 12, 48, 24, 40, 11 if kind == NEAR else None), 120
    a = Latent(ops, mix, dtype, t, portion=3)
    assert a.cache.ring == (13 if kind == NEAR else 128)
    for i in range(t):
        close(f"token {i}", a.ref[i], a.one(i, 1 + i % 3), dtype, exact=5e-6, half=1.5e-2)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("window", [5, 64, 71])
@pytest.mark.parametrize("inside", [True, False])
def test_a_key_at_the_edge_of_the_window(ops, dtype, window, inside):
    """The one key that matters is the oldest visible one, or the first that is not: in a portion and decoded."""
    mix, i = mixer(NEAR, 4, 64, 8, 32, 48, 56, window), 100
    j = i - window + (1 if inside else 0)
    for form in forms(ops, mix, dtype):
        a = Latent(ops, mix, dtype, i + 1, portion=60, spike=(i, j))
        wrong = a.plain(-1 if inside else 1)[i]
        assert float((wrong - a.ref[i]).pow(2).mean().sqrt()) > 0.3 * float(a.ref[i].pow(2).mean().sqrt())
        a.rows(0, 50, form)
        a.rows(50, 100, form)
        close("decoded", a.ref[i], a.one(i, 3), dtype, exact=1e-5, half=3e-2)
        close("portion", a.ref[i], a.rows(50, 101, form)[-1], dtype, exact=1e-5, half=3e-2)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("j", [0, 1, 63, 64, 129, 255, 256])
def test_a_key_far_away(ops, dtype, j):
    """One early key, hundreds of positions back, decides a late query; positions around the edges of key tiles."""
    mix, i = mixer(WIDE, 3, 48, 16, 24, 40, 64), 300
    a = Latent(ops, mix, dtype, i + 1, portion=150, spike=(i, j))
    wrong = a.plain(without=j)[i]
    assert float((wrong - a.ref[i]).pow(2).mean().sqrt()) > 0.3 * float(a.ref[i].pow(2).mean().sqrt())
    for form in forms(ops, mix, dtype):
        for lo in (0, 150):
            a.rows(lo, lo + 150, form)
        close("decoded", a.ref[i], a.one(i, 5), dtype, exact=1e-5, half=3e-2)
        close("portion", a.ref[i], a.rows(200, 301, form, 4)[-1], dtype, exact=1e-5, half=3e-2)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("sink", [-30.0, 0.0, 4.0, 60.0])
def test_sink(ops, dtype, sink):
    """From one that does not count to one that takes all of the weight; the very first tokens feel it most."""
    mix = mixer(NEAR, 5, 24, 8, 16, 24, 32, 12)
    for form in forms(ops, mix, dtype):
        a = Latent(ops, mix, dtype, 40, portion=33, sink=sink)
        close("first portion", a.ref[:33], a.rows(0, 33, form, 2), dtype, exact=1e-5, half=1.5e-2)
        close("token", a.ref[33], a.one(33, 2), dtype, exact=1e-5, half=1.5e-2)
        close("very first token", a.ref[0], a.one(0, 4), dtype, exact=1e-5, half=1.5e-2)


def test_bad_sizes_are_refused(ops):
    import tilert_b200 as tb
    from tilert_b200.kv_cache import LatentCache

    mix, pos = mixer(NEAR, 4, 32, 16, 32, 32, 32, 20), torch.zeros(1, dtype=I32, device="cuda")
    cache = LatentCache(32, 16, 20, 500, 10, "cuda", BF16)
    lat, part = torch.zeros(44, 64, device="cuda"), torch.zeros(44 * 34, device="cuda")
    with pytest.raises(tb.TilertError):  # the ring holds portions of ten
        ops.latent_attn(lat, cache, 11, mix, pos, 1, part)
    with pytest.raises(ValueError):
        ops.latent_attn(lat, cache, 10, mix, pos, 4, part)
    q, att = torch.zeros(11, 4, 48, dtype=BF16, device="cuda"), torch.zeros(11, 128, dtype=BF16, device="cuda")
    with pytest.raises(tb.TilertError):
        ops.expanded_attn(q, torch.zeros(29, 256, dtype=BF16, device="cuda"), cache, 11, mix, pos, None, None, True, att)
    with pytest.raises(tb.TilertError):
        ops.vec_gated(torch.zeros(8, device="cuda"), torch.zeros(2, 4, 8, dtype=BF16, device="cuda"), torch.zeros(4, device="cuda"), 4, 8, 1.0, ALPHA,
                      y=torch.zeros(8, device="cuda"))
