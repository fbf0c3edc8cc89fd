"""The mechanisms of ``include/tilert_gqa.h`` one by one against the plain restatement in ``oracle/ralasun.py``, in both
activation types, at sizes that are not multiples of anything convenient."""

import types

import pytest
import torch

from oracle import ralasun as R

pytestmark = pytest.mark.gpu

BF16, F32, I32, I64 = torch.bfloat16, torch.float32, torch.int32, torch.int64
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


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rnd(seed, *shape, std=1.0, dtype=F32):
    return (torch.randn(*shape, generator=gen(seed)) * std).to(dtype)


def padded(t, m=8, device="cuda"):
    """Rows padded with zeros to a multiple of m elements."""
    k = t.shape[-1]
    return torch.nn.functional.pad(t, (0, (k + m - 1) // m * m - k)).contiguous().to(device)


def close(name, ref, out, dtype, exact=2e-6, half=6e-3):
    ref, out = ref.double().cpu(), out.double().cpu()
    assert ref.shape == out.shape, (name, ref.shape, out.shape)
    err = ((ref - out).pow(2).mean().sqrt() / ref.pow(2).mean().sqrt().clamp_min(1e-30)).item()
    worst = ((ref - out).abs().max() / ref.abs().max().clamp_min(1e-30)).item()
    lim = exact if dtype == F32 else half
    assert err <= lim and worst <= 8 * lim, f"{name}: rms {err:.2e}, worst {worst:.2e}, limit {lim:.0e}"


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("dim", [50, 256])
def test_embedding_norm(ops, dtype, dim):
    table, w = rnd(0, 37, dim, std=3.0, dtype=BF16), rnd(1, dim, std=0.3)
    toks = torch.randint(0, 37, (11,), generator=gen(2))
    x = torch.zeros(11, ops.pad(dim), device="cuda")
    xh = torch.zeros(11, ops.pad(dim), dtype=dtype, device="cuda")
    ops.embed_norm(toks.cuda(), padded(table), padded(1 + w), 1e-3, dim, x, xh)
    ref = R.norm_around_one(table[toks].double(), w.double(), 1e-3)
    close("x", ref, x[:, :dim], F32)
    close("xh", ref, xh[:, :dim], dtype)
    assert float(x[:, dim:].abs().sum()) == 0


def test_a_token_outside_the_vocabulary_sets_the_status(ops):
    import tilert_b200 as tb

    x = torch.zeros(1, 16, device="cuda")
    ops.embed_norm(torch.tensor([5], device="cuda"), torch.zeros(5, 16, dtype=BF16, device="cuda"), torch.ones(16, device="cuda"),
                   1e-6, 16, x, None, exact=True)
    assert tb.device_status(0, "ralasun") == 4
    assert tb.device_status(0, "ralasun") == 0


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("shared", [False, True])
def test_residual_norm_of_a_row_and_of_combined_experts(ops, dtype, shared):
    dim, rows, top, eps = 75, 9, 3, 1e-2
    x0, y, w = rnd(0, rows, dim), rnd(1, rows, dim, std=2.0), rnd(2, dim, std=0.3)
    x, xh = padded(x0), torch.zeros(rows, ops.pad(dim), dtype=dtype, device="cuda")
    ops.residual_norm(x, xh, padded(1 + w), eps, dim, rows, y=padded(y))
    ref = x0.double() + R.norm_around_one(y.double(), w.double(), eps)
    close("dense", ref, x[:, :dim], F32)
    close("copy", ref, xh[:, :dim], dtype)

    ye, ysh = rnd(3, rows * top, dim, dtype=dtype), rnd(4, rows, dim, dtype=dtype) if shared else None
    slot = torch.randperm(rows * top, generator=gen(5)).view(rows, top)
    sw = torch.softmax(rnd(6, rows, top), -1)
    x = padded(x0)
    ops.residual_norm(x, xh, padded(1 + w), eps, dim, rows, experts=padded(ye), slot_row=slot.to(I32).cuda(), slot_w=sw.cuda(),
                      shared=None if ysh is None else padded(ysh))
    comb = (ye.double()[slot] * sw.double()[..., None]).sum(1) + (0 if ysh is None else ysh.double())
    close("experts", x0.double() + R.norm_around_one(comb, w.double(), eps), x[:, :dim], F32)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("rows,n,k", [(1, 7, 24), (3, 130, 40), (70, 257, 200), (129, 96, 77), (300, 640, 512), (1000, 2500, 136)])
def test_product(ops, dtype, rows, n, k):
    x, w, b = rnd(0, rows, k, dtype=dtype), rnd(1, n, k, std=k ** -0.5, dtype=BF16), rnd(2, n)
    ref = x.double() @ w.double().T + b.double()
    out = torch.full((rows, n + 3), 7.0, device="cuda")
    ops.gemm(padded(x), padded(w), out, rows, n, k, bias=b.cuda())
    close("f32 out", ref, out[:, :n], F32, exact=3e-6)
    assert bool((out[:, n:] == 7.0).all())
    for ld in (n + n % 2 + 2, n + n % 2 + 3):  # pairs of features in one store, and one by one
        out = torch.full((rows, ld), 7.0, dtype=dtype, device="cuda")
        ops.gemm(padded(x), padded(w), out, rows, n, k, bias=b.cuda())
        close("same type out", ref, out[:, :n], dtype, exact=3e-6)
        assert bool((out[:, n:] == 7.0).all())


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("rows,ff,k", [(2, 5, 24), (90, 136, 72), (260, 200, 330), (700, 1300, 256)])
def test_gated_product(ops, dtype, rows, ff, k):
    x, g, u = rnd(0, rows, k, dtype=dtype), rnd(1, ff, k, std=2 * k ** -0.5, dtype=BF16), rnd(2, ff, k, std=2 * k ** -0.5, dtype=BF16)
    out = torch.zeros(rows, ops.pad(ff), dtype=dtype, device="cuda")
    ops.gemm(padded(x), padded(torch.stack([g, u])), out, rows, ff, k, gated=(1.25, ALPHA))
    ref = R.gated_unit(x.double() @ g.double().T, x.double() @ u.double().T, 1.25)
    close("gated", ref, out[:, :ff], dtype)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("counts", [[3, 0, 5, 1, 0, 90, 2], [0, 0, 4], [200, 130, 257, 1], [5]])
def test_grouped_products(ops, dtype, counts):
    n, k, e, rows = 150, 88, len(counts), sum(counts)
    x, w = rnd(0, rows, k, dtype=dtype), rnd(1, e, 2, n, k, std=k ** -0.5, dtype=BF16)
    c = torch.tensor(counts, dtype=I32, device="cuda")
    out, plain = (torch.zeros(rows + 2, n + 2, dtype=dtype, device="cuda") for _ in range(2))
    ops.gemm(padded(x), padded(w), out, rows, n, k, gated=(0.8, ALPHA), n_groups=e, counts=c)
    ops.gemm(padded(x), padded(w[:, 1]), plain, rows, n, k, n_groups=e, counts=c)
    r0 = 0
    for i, cnt in enumerate(counts):
        xs = x[r0: r0 + cnt].double()
        if cnt:
            g, u = xs @ w[i, 0].double().T, xs @ w[i, 1].double().T
            close(f"gated group {i}", R.gated_unit(g, u, 0.8), out[r0: r0 + cnt, :n], dtype)
            close(f"group {i}", u, plain[r0: r0 + cnt, :n], dtype, exact=3e-6)
        r0 += cnt
    assert float(out[rows:].abs().sum()) == 0 and float(out[:, n:].abs().sum()) == 0


@pytest.mark.parametrize("n_experts,top", [(5, 1), (33, 4), (200, 8), (7, 7)])
def test_routing_and_gather(ops, n_experts, top):
    rows, dim = 77, 40
    z = rnd(0, rows, n_experts, std=2.0)
    ids, rank, slot = (torch.zeros(rows, top, dtype=I32, device="cuda") for _ in range(3))
    w, counts = torch.zeros(rows, top, device="cuda"), torch.full((n_experts,), 9, dtype=I32, device="cuda")
    ops.route_rows(padded(z), rows, n_experts, top, ids, w, rank, counts)
    eye, zero = torch.eye(n_experts, dtype=torch.float64), torch.zeros(n_experts, dtype=torch.float64)
    for t in range(rows):
        ri, rw = R.route(z[t].double(), eye, zero, top)
        assert ids[t].tolist() == ri
        assert torch.allclose(w[t].cpu().double(), rw, atol=1e-6)
    flat = ids.flatten().long().cpu()
    assert torch.equal(counts.cpu().long(), torch.bincount(flat, minlength=n_experts))
    for e in range(n_experts):
        assert sorted(rank.flatten().cpu()[flat == e].tolist()) == list(range(int((flat == e).sum())))
    for dtype in TYPES:
        x = rnd(1, rows, dim, dtype=dtype)
        xs = torch.zeros(rows * top, ops.pad(dim), dtype=dtype, device="cuda")
        ops.gather_rows(padded(x), rows, dim, n_experts, top, ids, rank, counts, xs, slot)
        assert sorted(slot.flatten().tolist()) == list(range(rows * top))
        base = torch.cumsum(torch.bincount(flat, minlength=n_experts), 0)
        s = slot.cpu().long()
        for t in range(rows):
            for j in range(top):
                assert s[t, j] < base[flat.view(rows, top)[t, j]] and torch.equal(xs[s[t, j], :dim].cpu(), x[t])


# ------------------------------------------------------------------ attention
def mix_of(heads, kv_heads, dim, vdim, window, scale=None):
    return types.SimpleNamespace(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, window=window, scale=scale or dim ** -0.5)


def cache_of(mix, dtype, max_len, portion):
    from tilert_b200.kv_cache import RingKVCache

    return RingKVCache(mix.kv_heads, mix.dim, mix.vdim, mix.window, max_len, portion, "cuda", dtype)


class Attn:
    """Random projections of a sequence, the plain result, and the two launch forms over one cache."""

    def __init__(self, ops, mix, dtype, t, portion, seed=0, v_mode=0, spike=None):
        self.ops, self.mix, self.dtype, self.v_mode, self.eps = ops, mix, dtype, v_mode, 1e-5
        nq, nk, nv = mix.heads * mix.dim, mix.kv_heads * mix.dim, mix.kv_heads * mix.vdim
        self.qkv = rnd(seed, t, nq + nk + nv)
        self.qg, self.kg = rnd(seed + 1, nq, std=0.2) + 1, rnd(seed + 2, nk, std=0.2) + 1
        if spike is not None:  # one query and one key along the same direction: their score stands out by far
            i, j = spike
            d = rnd(seed + 3, mix.dim)
            self.qkv[i, :nq] = d.repeat(mix.heads) * 4
            self.qkv[j, nq: nq + nk] = d.repeat(mix.kv_heads) * 4
            self.qkv[j, nq + nk:] = 5.0
        self.lam, self.first = torch.tensor([0.3]), rnd(seed + 4, t, nv)
        q, k, v = (p.double() for p in self.qkv.split([nq, nk, nv], dim=-1))
        if v_mode == 2:
            v = R.mix_values(v, self.first.double(), 0.3)
        self.k = R.projection_norm(k, self.kg.double(), self.eps).view(t, mix.kv_heads, mix.dim)
        self.q = R.projection_norm(q, self.qg.double(), self.eps).view(t, mix.heads, mix.dim)
        self.v = v.view(t, mix.kv_heads, mix.vdim)
        self.ref = R.attend(self.q, self.k, self.v, mix.heads, mix.kv_heads, mix.scale, mix.window).flatten(1)
        self.cache = cache_of(mix, dtype, t + 8, portion)
        # what an earlier sequence left behind must not be seen
        self.cache.k.copy_(rnd(seed + 5, *self.cache.k.shape, std=3.0))
        self.cache.v.copy_(rnd(seed + 6, *self.cache.v.shape, std=9.0))
        self.cache.k[..., mix.dim:] = 0
        self.cache.v[..., mix.vdim:] = 0
        self.dev = [t_.cuda() for t_ in (self.qkv, self.qg, self.kg, self.lam, self.first)]
        self.pos = torch.zeros(1, dtype=I32, device="cuda")

    def rows(self, lo, hi):
        ops, mix, n = self.ops, self.mix, hi - lo
        qkv, qg, kg, lam, first = self.dev
        self.pos.fill_(lo)
        q = torch.zeros(n, mix.heads, ops.pad(mix.dim, 16), dtype=self.dtype, device="cuda")
        f = first[lo:hi].contiguous()
        ops.qkv_rows(qkv[lo:hi].contiguous(), qg, kg, self.eps, self.v_mode, lam, f, n, mix, self.cache, self.pos, q)
        out = torch.zeros(n, ops.pad(mix.heads * mix.vdim), dtype=self.dtype, device="cuda")
        ops.attn_rows(q, mix, self.cache, self.pos, n, out)
        return out[:, : mix.heads * mix.vdim], f

    def one(self, i, n_splits):
        ops, mix = self.ops, self.mix
        qkv, qg, kg, lam, first = self.dev
        self.pos.fill_(i)
        part = torch.zeros(mix.heads * n_splits * (ops.pad(mix.vdim, 16) + 2), device="cuda")
        counter = torch.zeros(ops.head_blocks(mix.heads, mix.kv_heads), dtype=I32, device="cuda")
        out, f = torch.zeros(mix.heads * mix.vdim, device="cuda"), first[i].contiguous()
        ops.vec_attn(qkv[i].contiguous(), qg, kg, self.eps, self.v_mode, lam, f, mix, self.cache, self.pos, n_splits, part, counter, out)
        assert int(counter.abs().sum()) == 0
        return out, f


SHAPES = [(4, 2, 32, 32, 20), (6, 1, 40, 24, 65), (5, 5, 96, 64, 64), (20, 1, 24, 136, 7), (8, 2, 128, 256, 130), (12, 4, 72, 72, None),
          (3, 1, 17, 9, 1), (2, 2, 272, 300, 30)]


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("shape", SHAPES)
def test_attention_in_portions_and_token_by_token(ops, dtype, shape):
    mix, t = mix_of(*shape), 150
    a = Attn(ops, mix, dtype, t, portion=70)
    lo = 0
    for n in (64, 2, 70, 3):
        out, _ = a.rows(lo, lo + n)
        close(f"portion at {lo}", a.ref[lo: lo + n], out, dtype, exact=3e-6, half=1e-2)
        lo += n
    for i, s in zip(range(lo, t), (1, 2, 5, 1, 3, 40, 1, 2, 4, 7, 8)):
        out, _ = a.one(i, s)
        close(f"token {i}, {s} splits", a.ref[i], out, dtype, exact=3e-6, half=1e-2)


@pytest.mark.parametrize("dtype", TYPES)
def test_decoding_past_many_turns_of_the_ring(ops, dtype):
    mix, t = mix_of(4, 2, 32, 48, 11), 120
    a = Attn(ops, mix, dtype, t, portion=3)  # ring of 13 rows
    assert a.cache.ring == 13
    for i in range(t):
        out, _ = a.one(i, 1 + i % 3)
        close(f"token {i}", a.ref[i], out, dtype, exact=3e-6, half=1e-2)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("window", [5, 64, 71])
@pytest.mark.parametrize("inside", [True, False])
def test_a_key_at_the_edge_of_the_window(ops, dtype, window, inside):
    """The one key that matters is the oldest visible one, or the first that is not: in a portion and decoded."""
    mix, i = mix_of(4, 2, 64, 32, window, scale=0.5), 100
    j = i - window + (1 if inside else 0)
    a = Attn(ops, mix, dtype, i + 1, portion=60, spike=(i, j))
    other = Attn(ops, mix, dtype, i + 1, portion=60)
    moved = float((a.ref[i] - other.ref[i]).abs().mean())
    assert (moved > 1.0) if inside else True
    a.rows(0, 50)
    a.rows(50, 100)
    out, _ = a.one(i, 3)
    close("decoded", a.ref[i], out, dtype, exact=3e-6, half=2e-2)
    out, _ = a.rows(50, 101)  # the same positions again, now with the query inside the portion
    close("portion", a.ref[i], out[-1], dtype, exact=3e-6, half=2e-2)
    assert (float(out[-1].float().mean()) > 4.5) == inside


@pytest.mark.parametrize("dtype", TYPES)
def test_value_mixing(ops, dtype):
    mix = mix_of(4, 2, 32, 24, 16)
    for mode in (0, 1, 2):
        a = Attn(ops, mix, dtype, 40, portion=33, v_mode=mode)
        out, f = a.rows(0, 33)
        close(f"mode {mode}", a.ref[:33], out, dtype, exact=3e-6, half=1e-2)
        nv = mix.kv_heads * mix.vdim
        want = a.qkv[:33, -nv:] if mode == 1 else a.first[:33]
        assert torch.equal(f.cpu(), want)
        out, f = a.one(33, 2)
        close(f"mode {mode} token", a.ref[33], out, dtype, exact=3e-6, half=1e-2)
        assert torch.equal(f.cpu(), a.qkv[33, -nv:] if mode == 1 else a.first[33])


def test_a_cache_too_small_for_the_portion_is_refused(ops):
    import tilert_b200 as tb

    mix = mix_of(4, 2, 32, 32, 20)
    cache = cache_of(mix, BF16, 500, 10)
    q, out = torch.zeros(11, 4, 32, dtype=BF16, device="cuda"), torch.zeros(11, 128, dtype=BF16, device="cuda")
    with pytest.raises(tb.TilertError):
        ops.attn_rows(q, mix, cache, torch.zeros(1, dtype=I32, device="cuda"), 11, out)


# ------------------------------------------------------------------ one-token products
@pytest.mark.parametrize("n,k", [(1, 8), (5, 30), (150, 200), (777, 4096), (300, 9000), (40000, 136), (64, 17000)])
def test_one_token_product_with_its_norms(ops, n, k):
    eps = 1e-3
    x, y, g1, g2 = rnd(0, k), rnd(1, k, std=3.0), rnd(2, k, std=0.3), rnd(3, k, std=0.3)
    w, b = rnd(4, n, k, std=k ** -0.5, dtype=BF16), rnd(5, n)
    wd, out, xo = padded(w), torch.zeros(n, device="cuda"), torch.zeros(ops.pad(k), device="cuda")
    ops.vec_dense(padded(x), wd, out, n, k, bias=b.cuda())
    close("plain", w.double() @ x.double() + b.double(), out, F32, exact=5e-6)
    ops.vec_dense(padded(x), wd, out, n, k, y=padded(y), gain=padded(1 + g1), eps=eps, x_out=xo)
    v = x.double() + R.norm_around_one(y.double(), g1.double(), eps)
    close("residual", v, xo[:k], F32)
    close("norm and residual", w.double() @ v, out, F32, exact=5e-6)
    ops.vec_dense(padded(x), wd, out, n, k, y=padded(y), gain=padded(1 + g1), gain2=padded(1 + g2), eps=eps)
    close("and a norm on top", w.double() @ R.norm_around_one(v, g2.double(), eps), out, F32, exact=5e-6)
    ops.vec_dense(padded(x), wd, out, n, k, gain2=padded(1 + g2), eps=eps)
    close("norm alone", w.double() @ R.norm_around_one(x.double(), g2.double(), eps), out, F32, exact=5e-6)


@pytest.mark.parametrize("dim,ff,ff_sh,n_experts,top", [(40, 12, 0, 5, 1), (200, 50, 90, 9, 3), (512, 300, 1024, 64, 8), (96, 40, 20, 4, 4),
                                                        (64, 9000, 64, 3, 2)])
def test_one_token_experts(ops, dim, ff, ff_sh, n_experts, top):
    mlp = {"router": {"top": top}, "expert": {"limit": 0.9}, "shared": {"limit": 1.4} if ff_sh else None}
    x = rnd(0, 1, dim)
    w = {"m.router": rnd(1, n_experts, dim, std=2 * dim ** -0.5, dtype=BF16), "m.router.b": rnd(2, n_experts)}
    for e in range(n_experts):
        for i, nm in enumerate(("gate", "up")):
            w[f"m.e{e}.{nm}"] = rnd(10 + 3 * e + i, ff, dim, std=2 * dim ** -0.5, dtype=BF16)
        w[f"m.e{e}.down"] = rnd(12 + 3 * e, dim, ff, std=ff ** -0.5, dtype=BF16)
    if ff_sh:
        w |= {"m.shared.gate": rnd(5, ff_sh, dim, std=2 * dim ** -0.5, dtype=BF16), "m.shared.up": rnd(6, ff_sh, dim, std=dim ** -0.5, dtype=BF16),
              "m.shared.down": rnd(7, dim, ff_sh, std=ff_sh ** -0.5, dtype=BF16)}
    wd = {k: v.double() for k, v in w.items()}
    ref = R.mixture(x.double(), wd, "m", mlp)[0]
    logits = (wd["m.router"] @ x[0].double() + wd["m.router.b"]).float()
    gu = padded(torch.stack([torch.stack([w[f"m.e{e}.gate"], w[f"m.e{e}.up"]]) for e in range(n_experts)]))
    dn = padded(torch.stack([w[f"m.e{e}.down"] for e in range(n_experts)]))
    sgu = padded(torch.stack([w["m.shared.gate"], w["m.shared.up"]])) if ff_sh else None
    sdn = padded(w["m.shared.down"]) if ff_sh else None
    hidden = torch.zeros(ops.pad(ff_sh) + top * ops.pad(ff), device="cuda")
    ids, sw, out = torch.zeros(top, dtype=I32, device="cuda"), torch.zeros(top, device="cuda"), torch.zeros(dim, device="cuda")
    ops.vec_gate_up(padded(x[0]), dim, logits.cuda(), top, gu, sgu, ff, ff_sh, 0.9, 1.4, ALPHA, hidden, ids, sw)
    ops.vec_down(hidden, ids, sw, top, dn, sdn, ff, ff_sh, dim, out)
    rid, rw = R.route(x[0].double(), wd["m.router"], wd["m.router.b"], top)
    assert ids.tolist() == rid and torch.allclose(sw.cpu().double(), rw, atol=1e-6)
    close("experts", ref, out, F32, exact=5e-6)


def test_sampling_of_this_library(ops):
    logits = rnd(0, 2, 900)
    tok, lp = torch.zeros(2, dtype=I32, device="cuda"), torch.zeros(2, device="cuda")
    ops.sample(logits.cuda(), torch.tensor([0.0, 1.0, 0.0, 0.0], device="cuda"), tok, token_logprob=lp)
    assert tok.tolist() == logits.argmax(-1).tolist()
    ref = torch.log_softmax(logits, -1).max(-1).values
    assert torch.allclose(lp.cpu(), ref, atol=1e-4)
