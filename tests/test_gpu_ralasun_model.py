"""Whole Ralasun models on the shared driver against the plain restatement: prompts whole and in portions, decoding
through the ring caches, sequences one after the other, generation, the command line and the trace runner."""

import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from oracle import ralasun as R
from ralasun_models import CONFIGS, case, check_rows, row_errors

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def tb():
    import tilert_b200

    tilert_b200.load_backend("ralasun")
    tilert_b200.tilert_init(0, "ralasun")
    yield tilert_b200
    assert tilert_b200.device_status(0, "ralasun") == 0


def model_of(name, dtype, n, **kw):
    from tilert_b200.models.ralasun.model import RalasunModel

    args, sd, toks, ref, taps, close = case(name, n)
    return RalasunModel(args, sd, "cuda", dtype, **kw), toks, ref, taps, close


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
    n = 128 if name == "one" else 160
    model, toks, ref, taps, close = model_of(name, dtype, n)
    model.layer_taps = []
    out = model.prefill(toks, list(range(n)))
    for i, (want, got) in enumerate(zip(taps, model.layer_taps)):
        e = (got.double().cpu() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
        assert float(e.median()) < (3e-6 if dtype == "float32" else 2e-2), f"layer {i}: {float(e.median()):.2e}"
    check_rows("prompt", dtype, ref, out, close)
    assert torch.equal(out[-1].argmax().cpu(), model.token_out.cpu()[0])
    if dtype == "float32":  # a subset, in any order of asking
        model.reset_sequence()
        some = model.prefill(toks, [3, 50, n - 1])
        assert torch.equal(some, out[[3, 50, n - 1]])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_token_by_token_and_in_portions(tb, name, dtype):
    n = 128 if name == "one" else 160
    model, toks, ref, _, close = model_of(name, dtype, n)
    for cuts in ([1], [2], [3, 1, 17, 2, 64, 5, 1], [n - 20, 1], [8], [33, 31, 1, 1, 40, 2]):
        check_rows(f"{name} in {cuts}", dtype, ref, run(model, toks, cuts), close)


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompts_longer_than_a_portion_and_long_decoding(tb, dtype):
    """Portions of 24 tokens make the rings turn many times in the prompt; then 150 decoded tokens."""
    n = 400
    model, toks, ref, _, close = model_of("open", dtype, n, portion=24)
    assert model.layers[0].cache.ring == 63 and model.layers[1].cache.ring == 420
    check_rows("small portions", dtype, ref, run(model, toks, [250, 1]), close)
    check_rows("portions inside a step", dtype, ref, run(model, toks, [190, 7, 120, 1]), close)


@pytest.mark.parametrize("dtype", DTYPES)
def test_sequences_one_after_the_other_do_not_see_each_other(tb, dtype):
    model, toks, ref, _, close = model_of("toy", dtype, 160)
    alone = run(model, toks[:90], [40, 3, 1])
    other = [(t * 7 + 3) % model.args.vocab_size for t in toks]
    run(model, other, [100, 1])
    again = run(model, toks[:90], [40, 3, 1])
    assert torch.equal(alone, again)
    check_rows("first request", dtype, ref[:90], again, close[:90])
    with pytest.raises(ValueError):
        model.forward(1, 3)  # the device position is 90
    model.reset_sequence()
    with pytest.raises(ValueError):
        model.prefill([1] * (model.args.max_seq_len + 1))


def test_a_window_that_is_one_off_shows(tb):
    """The comparison is sharp enough to tell a window from its neighbours (mistake planted in the restatement)."""
    model, toks, ref, _, close = model_of("toy", "float32", 160)
    args, sd, _, _, _, _ = case("toy", 160)
    out = run(model, toks, [100, 1])
    for delta in (-1, 1):
        cfg = args.to_config()
        cfg["layers"][0]["mixer"]["mask"]["size"] += delta
        wrong = R.forward(cfg, sd, toks, torch.float64)
        assert float(row_errors(wrong, out)[40:].median()) > 20 * float(row_errors(ref, out).max())


@pytest.mark.parametrize("name", ["toy", "open"])
def test_greedy_generation_through_the_generator(tb, name):
    from tilert_b200.models.ralasun.generator import RalasunGenerator

    model, toks, _, _, _ = model_of(name, "float32", 160)
    args, sd, _, _, _, _ = case(name, 160)
    prompt, n_new = toks[:50], 40
    gen = RalasunGenerator(model, max_new_tokens=n_new)
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
    model, toks, _, _, _ = model_of("toy", "bfloat16", 160)
    eager, _, _, _, _ = model_of("toy", "bfloat16", 160, use_graph=False)
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

    args, sd, _, _, _, _ = case(name, 128 if name == "one" else 160)
    d = tmp_path / "model"
    d.mkdir()
    (d / "config.json").write_text(json.dumps(args.to_config()))
    save_file({k: v.contiguous() for k, v in sd.items()}, str(d / "model.safetensors"))
    return d


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_runner_replays_requests(tb, tmp_path, dtype):
    d, out = _save(tmp_path, "uneven"), tmp_path / "out"
    out.mkdir()
    args, _, toks, ref, _, close = case("uneven", 160)
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
    p = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(d), "--dtype", dtype, "--out", str(out), "--max-tokens", "128"],
                       input="\n".join(json.dumps(s) for s in steps), capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [ln for ln in p.stdout.splitlines() if ln.startswith("done")] == [f"done {s['step']}" for s in steps]
    got = []
    for s, rows in want_rows.items():
        got.append(torch.frombuffer(bytearray((out / f"{s}.f32").read_bytes()), dtype=torch.float32).view(len(rows), -1))
    picked = [r for rows in want_rows.values() for r in rows]
    check_rows("trace", dtype, ref[picked], torch.cat(got), close[picked])
    assert not (out / "5.f32").exists()


def test_command_line_with_random_and_with_saved_weights(tb, tmp_path):
    d = _save(tmp_path, "toy")
    for extra in (["--model", "ralasun", "--use-random-weights", "--dtype", "float32"], ["--model-weights-dir", str(d)]):
        out = subprocess.run([sys.executable, "-m", "tilert_b200.generate", "--max-new-tokens", "8", "--prompt-len", "6", "--max-seq-len",
                              "128", *extra], cwd=ROOT, capture_output=True, text=True, timeout=600)
        assert out.returncode == 0, out.stderr[-2000:]
        assert "tokens/s" in out.stdout
