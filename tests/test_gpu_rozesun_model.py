"""Whole Rozesun models on the shared driver against the plain restatement: prompts whole and in portions, decoding
through the latent caches, sequences one after the other, generation, the command line and the trace runner."""

import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from oracle import rozesun as R
from ralasun_models import row_errors
from rozesun_models import CONFIGS, case, check_rows

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
DTYPES = ["float32", "bfloat16"]
N = {name: 128 if name == "one" else 160 for name in CONFIGS}


@pytest.fixture(scope="module")
def tb():
    import tilert_b200

    tilert_b200.load_backend("ralasun")
    tilert_b200.tilert_init(0, "ralasun")
    yield tilert_b200
    assert tilert_b200.device_status(0, "ralasun") == 0


def model_of(name, dtype, n=None, **kw):
    from tilert_b200.models.rozesun.model import RozesunModel

    args, sd, toks, ref, taps = case(name, n or N[name])
    return RozesunModel(args, sd, "cuda", dtype, **kw), toks, ref, taps


def run(model, toks, cuts):
    """The sequence in portions of the given sizes (the last size repeats); logits of every position."""
    model.reset_sequence()
    out, lo, i = [], 0, 0
    while lo < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - lo)
        out.append(model.prefill(toks[lo: lo + n], list(range(n))))
        lo, i = lo + n, i + 1
    return torch.cat(out)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_layer_by_layer(tb, name, dtype):
    model, toks, ref, taps = model_of(name, dtype)
    model.layer_taps = []
    out = model.prefill(toks, list(range(len(toks))))
    assert len(model.layer_taps) == len(taps)
    for i, (want, got) in enumerate(zip(taps, model.layer_taps)):
        e = (got.double().cpu() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
        assert float(e.median()) < (3e-6 if dtype == "float32" else 2e-2), f"layer run {i}: {float(e.median()):.2e}"
    check_rows("prompt", dtype, ref, out)
    assert torch.equal(out[-1].argmax().cpu(), model.token_out.cpu()[0])
    if dtype == "float32":  # a subset, in any order of asking
        model.reset_sequence()
        pick = [3, 50, len(toks) - 1]
        assert torch.equal(model.prefill(toks, pick), out[pick])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_token_by_token_and_in_portions(tb, name, dtype):
    model, toks, ref, _ = model_of(name, dtype)
    for cuts in ([1], [2], [3, 1, 17, 2, 64, 5, 1], [len(toks) - 20, 1], [8], [33, 31, 1, 1, 40, 2]):
        check_rows(f"{name} in {cuts}", dtype, ref, run(model, toks, cuts))


@pytest.mark.parametrize("form", ["absorbed", "expanded"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_either_form_of_the_attention(tb, name, form, monkeypatch):
    """The sizes alone choose the form; each is right for any of them."""
    from tilert_b200.models.rozesun import layer

    monkeypatch.setattr(layer, "expansion_pays", lambda *a: form == "expanded")
    model, toks, ref, _ = model_of(name, "bfloat16")
    for cuts in ([len(toks)], [2], [50, 7, 64, 3]):
        check_rows(f"{name} in {cuts}", "bfloat16", ref, run(model, toks, cuts))


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompts_longer_than_a_portion_and_long_decoding(tb, dtype):
    """Portions of 24 tokens make the rings turn many times in the prompt; then 150 decoded tokens."""
    model, toks, ref, _ = model_of("deep", dtype, 400, portion=24)
    assert [layer.caches[0].ring for layer in model.layers] == [63, 420, 153]
    check_rows("small portions", dtype, ref, run(model, toks, [250, 1]))
    check_rows("portions inside a step", dtype, ref, run(model, toks, [190, 7, 120, 1]))


@pytest.mark.parametrize("dtype", DTYPES)
def test_sequences_one_after_the_other_do_not_see_each_other(tb, dtype):
    model, toks, ref, _ = model_of("toy", dtype)
    alone = run(model, toks[:90], [40, 3, 1])
    run(model, [(t * 7 + 3) % model.args.vocab_size for t in toks], [100, 1])
    again = run(model, toks[:90], [40, 3, 1])
    assert torch.equal(alone, again)
    check_rows("first request", dtype, ref[:90], again)
    with pytest.raises(ValueError):
        model.forward(1, 3)  # the device position is 90
    model.reset_sequence()
    with pytest.raises(ValueError):
        model.prefill([1] * (model.args.max_seq_len + 1))


def test_every_pass_of_the_loop_has_its_own_cache(tb):
    model, toks, _, _ = model_of("uneven", "float32")
    run(model, toks[:30], [30])
    a, b, c = (cache.rows for cache in model.layers[0].caches)
    assert len(model.layers[2].caches) == 1 and len({t.data_ptr() for t in (a, b, c)}) == 3
    assert not torch.equal(a, b) and not torch.equal(b, c)


def _window(delta):
    def change(cfg, sd):
        cfg["layers"][0]["mixer"]["mask"]["size"] += delta
    return change


def _no_sink(cfg, sd):
    sd["l0.mix.sink"] = torch.full_like(sd["l0.mix.sink"], -1e4)


def _base(cfg, sd):
    cfg["layers"][1]["mixer"]["rot"]["base"] *= 1.01


def _no_step(cfg, sd):
    sd["loop.step"][1] = 0


def _times(cfg, sd):
    cfg["loop"]["times"] = 1


def _limit(cfg, sd):
    cfg["layers"][0]["mlp"]["limit"] *= 1.05


def _norm_bias(cfg, sd):
    sd["l1.norm2b.b"] = torch.zeros_like(sd["l1.norm2b.b"])


def _swap_pairs(cfg, sd):
    cfg["layers"][1]["type"] = "swapped"


@pytest.mark.parametrize("plant", [_window(-1), _window(1), _no_sink, _base, _no_step, _times, _limit, _norm_bias, _swap_pairs])
def test_the_comparison_shows_a_mistake(tb, plant, monkeypatch):
    """It is sharp enough to tell every mechanism from a near miss (planted in the restatement)."""
    monkeypatch.setitem(R.KINDS, "swapped", dict(interleaved=True, window=False, sink=False))
    model, toks, ref, _ = model_of("toy", "float32")
    args, sd, _, _, _ = case("toy", N["toy"])
    out = run(model, toks, [100, 1])
    cfg, sd = args.to_config(), {k: v.clone() for k, v in sd.items()}
    plant(cfg, sd)
    wrong = R.forward(cfg, sd, toks, torch.float64)
    assert float(row_errors(wrong, out)[40:].median()) > 20 * float(row_errors(ref, out).max())


@pytest.mark.parametrize("name", ["toy", "deep"])
def test_greedy_generation_through_the_generator(tb, name):
    from tilert_b200.models.rozesun.generator import RozesunGenerator

    model, toks, _, _ = model_of(name, "float32")
    args, sd, _, _, _ = case(name, N[name])
    prompt, n_new = toks[:50], 40
    gen = RozesunGenerator(model, max_new_tokens=n_new)
    text, times, _, plen = gen.generate("", print_log=False, prompt_tokens=prompt)
    got = [int(t) for t in text.split()]
    assert plen == 50 and len(got) == n_new and len(times) == n_new
    ref = R.forward(args.to_config(), sd, prompt + got, torch.float64)
    for i, t in enumerate(got):
        row = ref[len(prompt) + i - 1]
        assert float(row.max() - row[t]) < 1e-3 * float(row.std()), (i, t)
    direct, logits = model.generate(prompt, n_new, collect_logits=True)
    assert direct == got and len(logits) == n_new
    gen.eos_id = got[5]
    assert [int(t) for t in gen.generate("", print_log=False, prompt_tokens=prompt)[0].split()] == got[: got.index(got[5])]


def test_decode_with_and_without_graphs_and_sampling(tb):
    model, toks, _, _ = model_of("toy", "bfloat16")
    eager, _, _, _ = model_of("toy", "bfloat16", use_graph=False)
    assert torch.equal(run(model, toks, [60, 1]), run(eager, toks, [60, 1]))
    model.set_sampling(0.8, 0.9, 50, True, seed=3)
    a = model.generate(toks[:20], 12)
    model.sample_step.zero_()
    assert a == model.generate(toks[:20], 12)
    assert float(model.token_logprob) < 0 and int(model.topn_indices[0, 0]) >= 0
    model.set_sampling(0.0)
    assert model.generate(toks[:20], 6) == eager.generate(toks[:20], 6)


def _save(tmp_path, name):
    from safetensors.torch import save_file

    args, sd, _, _, _ = case(name, N[name])
    d = tmp_path / "model"
    d.mkdir()
    (d / "config.json").write_text(json.dumps(args.to_config()))
    save_file({k: v.contiguous() for k, v in sd.items()}, str(d / "model.safetensors"))
    return d


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_runner_replays_requests(tb, tmp_path, dtype):
    d, out = _save(tmp_path, "uneven"), tmp_path / "out"
    out.mkdir()
    _, _, toks, ref, _ = case("uneven", N["uneven"])
    steps, at, want_rows = [], 0, {}
    for n in (70, 2, 1, 1, 30):
        want = [0, n - 1] if n > 1 else [0]
        steps.append({"step": len(steps), "entries": [{"id": "a", "tokens": toks[at: at + n], "want": want}], "end": []})
        want_rows[len(steps) - 1] = [at + w for w in want]
        at += n
    steps[-1]["end"] = ["a"]
    steps.append({"step": len(steps), "entries": [{"id": "b", "tokens": toks[:5], "want": []}], "end": []})
    steps.append({"step": len(steps), "entries": [{"id": "b", "tokens": toks[5:9], "want": [3]}], "end": ["b"]})
    want_rows[len(steps) - 1] = [8]
    p = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(d), "--dtype", dtype, "--out", str(out), "--max-tokens", "104"],
                       input="\n".join(json.dumps(s) for s in steps), capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [ln for ln in p.stdout.splitlines() if ln.startswith("done")] == [f"done {s['step']}" for s in steps]
    got = [torch.frombuffer(bytearray((out / f"{s}.f32").read_bytes()), dtype=torch.float32).view(len(rows), -1) for s, rows in want_rows.items()]
    check_rows("trace", dtype, ref[[r for rows in want_rows.values() for r in rows]], torch.cat(got))
    assert not (out / "5.f32").exists()


def test_command_line_with_random_and_with_saved_weights(tb, tmp_path):
    d = _save(tmp_path, "toy")
    for extra in (["--model", "rozesun", "--use-random-weights", "--dtype", "float32"], ["--model-weights-dir", str(d)]):
        out = subprocess.run([sys.executable, "-m", "tilert_b200.generate", "--max-new-tokens", "8", "--prompt-len", "6", "--max-seq-len",
                              "128", *extra], cwd=ROOT, capture_output=True, text=True, timeout=600)
        assert out.returncode == 0, out.stderr[-2000:]
        assert "tokens/s" in out.stdout
