"""Host side of the Rozesun design, without a GPU: the restatement's own consistency, configuration, weights, registry,
cache sizes and the choice of the attention's form."""

import json

import pytest
import torch

from oracle import rozesun as R
from ralasun_models import row_errors
from rozesun_models import CONFIGS, case
from tilert_b200 import gqa_ops, synthetic
from tilert_b200.kv_cache import LatentCache
from tilert_b200.models import registry
from tilert_b200.models.rozesun.layer import LayerWeights, expansion_pays
from tilert_b200.models.rozesun.model_args import MixerArgs, RozesunArgs

F64 = torch.float64


def test_restatement_mechanisms_by_hand():
    x = torch.tensor([[1.0, 3.0]], dtype=F64)
    w, b = torch.tensor([2.0, 1.0], dtype=F64), torch.tensor([0.5, 0.0], dtype=F64)
    assert torch.allclose(R.layer_norm(x, w, b, 0.0), torch.tensor([[-1.5, 1.0]], dtype=F64))
    assert torch.allclose(R.layer_norm(x, w, b, 3.0), torch.tensor([[-0.5, 0.5]], dtype=F64))
    v = torch.tensor([1.0, 0.0, 0.0, 2.0, 7.0], dtype=F64)
    c0, s0, c1, s1 = (f(torch.tensor(a, dtype=F64)) for a in (3.0, 3.0 * 16.0 ** -0.5) for f in (torch.cos, torch.sin))
    assert torch.allclose(R.rotate(v, 3, 16.0, 4, True), torch.stack([c0, s0, -2 * s1, 2 * c1, v[4]]))
    assert torch.allclose(R.rotate(v, 3, 16.0, 4, False), torch.stack([c0, -2 * s1, s0, 2 * c1, v[4]]))
    s = torch.log(torch.tensor([1.0, 3.0], dtype=F64))
    assert torch.allclose(R.sink_softmax(s, None), torch.tensor([0.25, 0.75], dtype=F64))
    assert torch.allclose(R.sink_softmax(s, torch.log(torch.tensor(4.0, dtype=F64))), torch.tensor([0.125, 0.375], dtype=F64))
    o = torch.ones(1, 2, 3, dtype=F64)
    assert torch.allclose(R.gate(o, torch.tensor([[0.0, 100.0]], dtype=F64)), torch.tensor([[0.5] * 3 + [1.0] * 3], dtype=F64))
    assert torch.allclose(R.gate(o, torch.tensor([[0.0, 100.0, 0, 0, 0, 100.0]], dtype=F64)), torch.tensor([[0.5, 1, 0.5, 0.5, 0.5, 1]], dtype=F64))
    assert R.runs(4, {"start": 1, "stop": 3, "times": 2}) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert R.runs(2, None) == [(0, None), (1, None)]


def test_restatement_scores_depend_on_distances():
    """Turning both sides by the same number of positions changes no score."""
    q, k = torch.randn(2, 8, dtype=F64, generator=torch.Generator().manual_seed(0))
    for inter in (False, True):
        scores = [R.rotate(q, p + 5, 100.0, 8, inter) @ R.rotate(k, p, 100.0, 8, inter) for p in (0, 1, 77)]
        assert torch.allclose(scores[0], scores[1]) and torch.allclose(scores[0], scores[2])
        assert not torch.allclose(scores[0], R.rotate(q, 6, 100.0, 8, inter) @ R.rotate(k, 0, 100.0, 8, inter))


def test_restatement_is_causal_and_windowed():
    args, sd, toks, ref, _ = case("one", 96)
    changed = list(toks)
    changed[20] = (changed[20] + 1) % args.vocab_size
    diff = row_errors(ref, R.forward(args.to_config(), sd, changed, F64))
    assert float(diff[:20].max()) == 0 and float(diff[20]) > 1e-3
    reach = 2 * sum(layer.mixer.window - 1 for layer in args.layers)  # two passes
    assert float(diff[20 + reach]) > 0 and float(diff[21 + reach:].max()) == 0


@pytest.mark.parametrize("name", list(CONFIGS))
def test_configuration_round_trip_and_order(name):
    args = CONFIGS[name]()
    assert RozesunArgs.from_config(json.loads(json.dumps(args.to_config())), args.max_seq_len) == args
    assert args.runs() == R.runs(len(args.layers), args.to_config()["loop"])


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("expanded", [True, False])
def test_weights_as_the_kernels_want_them(name, expanded):
    args = CONFIGS[name]()
    sd = synthetic.random_rozesun_state_dict(args, seed=1)
    for li, layer in enumerate(args.layers):
        m, w, p = layer.mixer, LayerWeights(args, sd, li, "cpu", expanded), f"l{li}.mix"
        d = args.dim
        assert torch.equal(w.z[: m.q_rank, :d], sd[f"{p}.dq"]) and torch.equal(w.z[w.off_c: w.off_c + m.kv_rank, :d], sd[f"{p}.dkv"][: m.kv_rank])
        assert torch.equal(w.z[w.off_r: w.off_r + m.rot_dim, :d], sd[f"{p}.dkv"][m.kv_rank:])
        assert torch.equal(w.z[w.off_g: w.off_g + m.gate_rows, :d], sd[f"{p}.g"])
        assert all(o % 8 == 0 for o in (w.off_c, w.off_r, w.off_g))
        ldh, dim8 = gqa_ops.pad(m.dim) + gqa_ops.pad(m.rot_dim), gqa_ops.pad(m.dim)
        uq, ref = w.uq.view(m.heads, ldh, -1)[..., : m.q_rank], sd[f"{p}.uq"].view(m.heads, m.dim + m.rot_dim, m.q_rank)
        assert torch.equal(uq[:, : m.dim], ref[:, : m.dim]) and torch.equal(uq[:, dim8: dim8 + m.rot_dim], ref[:, m.dim:])
        assert float(uq.float().abs().sum()) == pytest.approx(float(ref.float().abs().sum()), rel=1e-6)  # the rest is zero
        h = m.heads - 1
        assert torch.equal(w.uk_t[h, :, : m.dim], sd[f"{p}.uk"].view(m.heads, m.dim, -1)[h].T)
        assert torch.equal(w.uv[h, :, : m.kv_rank], sd[f"{p}.uv"].view(m.heads, m.vdim, -1)[h])
        assert (w.kv is not None) == expanded and (w.sink is not None) == m.sink and (w.down is None) == (layer.mlp is None)
        if expanded:
            dp, vp = gqa_ops.pad(m.dim, 16), gqa_ops.pad(m.vdim, 16)
            k, v = w.kv[: m.heads * dp].view(m.heads, dp, -1), w.kv[m.heads * dp:].view(m.heads, vp, -1)
            assert torch.equal(k[h, : m.dim, : m.kv_rank].T, w.uk_t[h, :, : m.dim]) and torch.equal(v[h, : m.vdim], w.uv[h])
            assert float(k[:, m.dim:].float().abs().sum()) == 0 and float(v[:, m.vdim:].float().abs().sum()) == 0
        assert torch.equal(w.norm1.bias[:d], sd[f"l{li}.norm1.b"].float()) and w.norm1.centered
        assert w.weight_bytes() >= 2 * sum(sd[f"{p}.{n}"].numel() for n in ("dq", "uq", "dkv", "uk", "uv", "g", "o"))


def test_bad_configurations_and_weights_are_refused():
    cfg = CONFIGS["toy"]().to_config()

    def refused(change):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(ValueError):
            RozesunArgs.from_config(bad)

    refused(lambda c: c["layers"][0].update(type="something else"))
    refused(lambda c: c["layers"][0]["mixer"].pop("mask"))
    refused(lambda c: c["layers"][0]["mixer"]["mask"].update(size=0))
    refused(lambda c: c["layers"][1]["mixer"].update(mask={"size": 5}))
    refused(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=8))
    refused(lambda c: c["layers"][1]["mixer"].update(rot_dim=3, rot={"base": 10.0, "dims": 3}))
    refused(lambda c: c["layers"][1]["mlp"].update(kind="other"))
    for loop in ({"start": 1, "stop": 1, "times": 2}, {"start": 0, "stop": 5, "times": 2}, {"start": 0, "stop": 2, "times": 0}):
        refused(lambda c, lp=loop: c.update(loop=lp))
    args = CONFIGS["uneven"]()
    for name in ("l0.mix.g", "l1.mix.uk", "l1.mlp.down", "l0.mix.sink"):
        sd = synthetic.random_rozesun_state_dict(args)
        sd[name] = sd[name][:2]
        with pytest.raises(ValueError):
            LayerWeights(args, sd, int(name[1]), "cpu", False)


def test_registry_chooses_by_configuration(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(CONFIGS["one"]().to_config()))
    f = registry.family_of_dir(tmp_path)
    assert f.name == "rozesun" and "float32" in f.dtypes and f is registry.family_of_preset("rozesun")


def test_cache_rows_and_rings():
    c = LatentCache(45, 14, 20, 500, 64, "cpu", torch.float32)
    assert c.rows.shape == (83, 64) and c.rows.shape[1] == gqa_ops.latent_row_len(45, 14) and c.bytes() == 83 * 64 * 4
    assert c.visible(7) == 7 and c.visible(400) == 20 and c.visible(400, 10) == 29 and c.visible(25, 10) == 25
    c = LatentCache(48, 16, None, 500, 64, "cpu", torch.bfloat16)
    assert c.rows.shape == (500, 64) and c.window == 0 and c.visible(321, 5) == 321


def test_the_form_of_the_attention_follows_the_work():
    m = MixerArgs("latent_attention", heads=16, dim=128, rot_dim=64, vdim=128, q_rank=512, kv_rank=512, scale=0.1, rot_base=1e4)
    assert not expansion_pays(m, 2, 4000, 4000) and expansion_pays(m, 2000, 2000, 2000)


def test_rotation_table():
    t = gqa_ops.rotation_table(300.0, 6, 50, "cpu")
    a = torch.tensor([49 * 300.0 ** (-2 * i / 6) for i in range(3)], dtype=F64)
    assert t.shape == (50, 6) and torch.allclose(t[49].double(), torch.cat([torch.cos(a), torch.sin(a)]), atol=1e-7)
