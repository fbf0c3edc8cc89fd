"""Host side of the Ralasun design, without a GPU: the restatement's own consistency, configuration, registry, ring
sizes, the shared driver's portions and the trace runner's bookkeeping."""

import io
import json

import pytest
import torch

from oracle import ralasun as R
from ralasun_models import CONFIGS, case, row_errors
from tilert_b200 import _cabi, build, synthetic
from tilert_b200.kv_cache import RingKVCache
from tilert_b200.models import registry
from tilert_b200.models.driver import SequenceDriver
from tilert_b200.models.generator import SequenceGenerator
from tilert_b200.models.ralasun.layer import LayerWeights
from tilert_b200.models.ralasun.model_args import RalasunArgs


def test_restatement_mechanisms_by_hand():
    x = torch.tensor([[3.0, 4.0]], dtype=torch.float64)
    assert torch.allclose(R.rms(x, 0.0), x / (12.5 ** 0.5))
    assert torch.allclose(R.norm_around_one(x, torch.tensor([0.0, 1.0], dtype=torch.float64), 0.0), R.rms(x, 0.0) * torch.tensor([1.0, 2.0]))
    assert list(R.visible(7, 3)) == [5, 6, 7] and list(R.visible(1, 3)) == [0, 1] and list(R.visible(2, None)) == [0, 1, 2]
    one = torch.tensor(1.0, dtype=torch.float64)
    assert torch.allclose(R.gated_unit(5 * one, 9 * one, 1.0), 1 / (1 + torch.exp(-1.702 * one)) * 2)
    assert torch.allclose(R.gated_unit(-5 * one, -9 * one, 1.0), 0 * one)  # the gate has no lower limit, but u + 1 = 0
    ids, w = R.route(one.view(1), torch.tensor([[1.0], [3.0], [2.0]], dtype=torch.float64), torch.zeros(3, dtype=torch.float64), 2)
    assert ids == [1, 2] and torch.allclose(w, torch.softmax(torch.tensor([3.0, 2.0], dtype=torch.float64), 0))
    assert torch.allclose(R.mix_values(one, 3 * one, 0.25), 1.5 * one)


def test_restatement_is_causal_and_windowed():
    args, sd, toks, ref, _, _ = case("uneven", 160)
    changed = list(toks)
    changed[20] = (changed[20] + 1) % args.vocab_size
    diff = row_errors(ref[:80], R.forward(args.to_config(), sd, changed[:80], torch.float64))
    assert float(diff[:20].max()) == 0 and float(diff[20]) > 1e-3
    reach = sum(layer.mixer.window - 1 for layer in args.layers)
    far = R.forward(args.to_config(), sd, changed, torch.float64)
    assert 20 + reach < 160 and float(row_errors(ref, far)[20 + reach + 1:].max()) == 0


@pytest.mark.parametrize("name", list(CONFIGS))
def test_configuration_round_trip_and_weights(name):
    args = CONFIGS[name]()
    assert RalasunArgs.from_config(json.loads(json.dumps(args.to_config())), args.max_seq_len) == args
    sd = synthetic.random_ralasun_state_dict(args, seed=1)
    for li, layer in enumerate(args.layers):
        w = LayerWeights(args, sd, li, "cpu")
        m = layer.mixer
        assert w.qkv.shape[1] % 8 == 0 and w.o.shape == (args.dim, (m.heads * m.vdim + 7) // 8 * 8)
        assert torch.equal(w.qkv[: m.heads * m.dim, : args.dim], sd[f"l{li}.mix.q"])
        assert torch.equal(w.norm1[: args.dim], 1 + sd[f"l{li}.norm1"].float()) and float(w.norm1[args.dim:].abs().sum()) == 0
        if layer.mlp is None:
            assert w.gate_up is None
            continue
        e = layer.mlp.experts - 1
        assert torch.equal(w.gate_up[e, 1, :, : args.dim], sd[f"l{li}.mlp.e{e}.up"])
        assert torch.equal(w.down[e, :, : layer.mlp.ff], sd[f"l{li}.mlp.e{e}.down"]) and float(w.down[..., layer.mlp.ff:].abs().sum()) == 0
        assert (w.shared_down is None) == (layer.mlp.shared_ff == 0)


def test_bad_configurations_are_refused():
    cfg = CONFIGS["toy"]().to_config()
    for path, value in ((("heads",), 5), (("mask", "size"), 0), (("vdim",), 40)):
        bad = json.loads(json.dumps(cfg))
        node = bad["layers"][2]["mixer"]
        for p in path[:-1]:
            node = node[p]
        node[path[-1]] = value
        with pytest.raises(ValueError):
            RalasunArgs.from_config(bad)
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["type"] = "something else"
    with pytest.raises(ValueError):
        RalasunArgs.from_config(bad)
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["mlp"]["router"]["top"] = 99
    with pytest.raises(ValueError):
        RalasunArgs.from_config(bad)
    args = CONFIGS["uneven"]()
    sd = synthetic.random_ralasun_state_dict(args)
    sd["l0.mlp.router"] = sd["l0.mlp.router"][:2]
    with pytest.raises(ValueError):
        LayerWeights(args, sd, 0, "cpu")


def test_registry_chooses_by_configuration(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(CONFIGS["one"]().to_config()))
    f = registry.family_of_dir(tmp_path)
    assert f.name == "ralasun" and "float32" in f.dtypes and f.name in build.TARGETS
    (tmp_path / "config.json").write_text(json.dumps({"architectures": ["DeepseekV32ForCausalLM"], "num_hidden_layers": 3}))
    assert registry.family_of_dir(tmp_path).name == "deepseek_v3_2"
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "unknown"}))
    with pytest.raises(ValueError):
        registry.family_of_dir(tmp_path)
    assert registry.family_of_preset("toy").name == "deepseek_v3_2" and registry.family_of_preset("ralasun").name == "ralasun"


def test_ring_sizes():
    c = RingKVCache(2, 40, 24, 20, 500, 64, "cpu", torch.float32)
    assert (c.ring, c.window, c.k.shape, c.v.shape) == (83, 20, (2, 83, 48), (2, 83, 32))
    assert c.visible(7) == 7 and c.visible(400) == 20
    for window in (None, 500, 900):  # nothing is ever outside
        c = RingKVCache(2, 40, 24, window, 500, 64, "cpu", torch.float32)
        assert c.ring == 500 and c.window == 0 and c.visible(321) == 321


def test_both_libraries_build_and_export_their_headers():
    import tilert_b200

    for name, be in tilert_b200._BACKENDS.items():
        assert build.build(model_type=name).exists() and not build.needs_build(name)
        lib = tilert_b200.load_backend(name)
        protos = _cabi.parse_header(_cabi.header_path(be.header))
        assert len(protos) >= 20 and all(hasattr(lib, n) for n in protos)
    assert any(p.name == "topk_radix.cuh" for p in build.sources(build.TARGETS["ralasun"].src))


class Counting(SequenceDriver):
    """A driver without kernels: the logits of a step name the token and its position."""

    def __init__(self, limit=50):
        self._init_sequence("cpu", 8, use_graph=False)
        self.limit, self.steps = limit, []

    def position_limit(self):
        return self.limit

    def _graph_key(self, pos):
        return 0

    def _step_ops(self, key):
        self.steps.append((int(self.token), int(self.cur_pos)))
        self.logits.zero_()
        self.logits[0, 0, (int(self.token) + 1) % 8] = 1.0 + int(self.cur_pos)
        self._choose(self.logits.view(1, -1))
        self.cur_pos += 1


def test_shared_driver_positions_prefill_and_generation():
    m = Counting()
    rows = m.prefill([3, 4, 5], [0, 2])
    assert m.steps == [(3, 0), (4, 1), (5, 2)] and rows.shape == (2, 8) and float(rows[1, 6]) == 3.0
    with pytest.raises(ValueError):
        m.forward(1, 0)
    with pytest.raises(ValueError):
        m.set_cur_pos(50)
    assert m.generate([1, 2], 3) == [3, 4, 5] and m._pos == 4  # the last token is not run
    m.set_cur_pos(49)
    m.forward(1, 49)
    with pytest.raises(ValueError):
        m.forward(1, 50)


def test_shared_generator_loop():
    class Gen(SequenceGenerator):
        def __init__(self, m):
            self.m, self.max_new_tokens = m, 4

        def _max_len(self):
            return self.m.limit

        def _prompt(self, tokens, times):
            self.m.prefill(tokens)
            times.append(0.0)
            return int(self.m.token_out)

        def _next(self, token):
            self.m.forward(token, self.m._pos)
            return int(self.m.token_out)

        def _end_sequence(self):
            self.m.reset_sequence()

    g = Gen(Counting())
    text, times, _, plen = g._generate_plain([1, 2], False)
    assert text.split() == ["3", "4", "5", "6"] and plen == 2 and len(times) == 4
    g.eos_id = 5
    assert g._generate_plain([1, 2], False)[0].split() == ["3", "4"]
    g = Gen(Counting(limit=4))
    assert g._generate_plain([1, 2], False)[0].split() == ["3", "4"]
    with pytest.raises(ValueError):
        g._tokens_of("text", None)


def test_trace_runner_keeps_one_request_at_a_time():
    from tilert_b200.trace_run import TraceRunner

    m = Counting()
    r = TraceRunner(m)
    assert r.step([{"id": "a", "tokens": [1, 2], "want": [1]}], []).shape == (1, 8)
    assert r.step([{"id": "a", "tokens": [3], "want": []}], []) is None and m._pos == 3
    with pytest.raises(ValueError):
        r.step([{"id": "b", "tokens": [3], "want": []}], [])
    r.step([], ["a"])
    r.step([{"id": "b", "tokens": [5], "want": [0]}], ["b"])
    assert m._pos == 0 and m.steps[-1] == (5, 0)
    with pytest.raises(ValueError):
        r.step([], ["b"])


def test_trace_runner_refuses_a_type_the_family_does_not_run_in(tmp_path, monkeypatch, capsys):
    from tilert_b200 import trace_run

    (tmp_path / "config.json").write_text(json.dumps({"architecture": "deepseek_v3_2"}))
    monkeypatch.setattr("sys.stdin", io.StringIO(""))
    assert trace_run.main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path)]) == 3
    assert "float32" in capsys.readouterr().err
