"""The model families: how a configuration is recognised and read, which native library carries the kernels, how a
model or a generator is made.  Entry points (the command line, the trace runner) choose a family here and nowhere
else."""

from __future__ import annotations

import json
from collections.abc import Callable
from dataclasses import dataclass, replace
from pathlib import Path


@dataclass(frozen=True)
class ModelFamily:
    name: str
    backend: str                       # native library with its kernels (tilert_b200.load_backend, build.TARGETS)
    architectures: tuple[str, ...]     # values of "architecture" / "architectures" / "model_type" in config.json
    dtypes: tuple[str, ...]            # activation types the family runs in
    load: Callable                     # (model_dir, device, dtype, max_seq_len) -> a SequenceDriver
    generator: Callable                # (model_dir or None, cli options) -> a SequenceGenerator
    presets: tuple[str, ...] = ()      # random-weight models of the command line


def _ralasun_load(model_dir, device, dtype, max_seq_len):
    from .ralasun.model import RalasunModel

    return RalasunModel.from_pretrained(model_dir, device, dtype, max_seq_len)


def _ralasun_generator(model_dir, o):
    from tilert_b200 import synthetic

    from .ralasun.generator import RalasunGenerator
    from .ralasun.model import RalasunModel
    from .ralasun.model_args import toy_args

    if model_dir is None:
        args = toy_args(o.max_seq_len)
        model = RalasunModel(args, synthetic.random_ralasun_state_dict(args, seed=o.seed), dtype=o.dtype)
    else:
        model = _ralasun_load(model_dir, "cuda", o.dtype, o.max_seq_len)
    return RalasunGenerator(model, o.max_new_tokens, sampling_seed=o.seed)


def _rozesun_load(model_dir, device, dtype, max_seq_len):
    from .rozesun.model import RozesunModel

    return RozesunModel.from_pretrained(model_dir, device, dtype, max_seq_len)


def _rozesun_generator(model_dir, o):
    from tilert_b200 import synthetic

    from .rozesun.generator import RozesunGenerator
    from .rozesun.model import RozesunModel
    from .rozesun.model_args import toy_args

    if model_dir is None:
        args = toy_args(o.max_seq_len)
        model = RozesunModel(args, synthetic.random_rozesun_state_dict(args, seed=o.seed), dtype=o.dtype)
    else:
        model = _rozesun_load(model_dir, "cuda", o.dtype, o.max_seq_len)
    return RozesunGenerator(model, o.max_new_tokens, sampling_seed=o.seed)


def _dsv32_args(model_dir, max_seq_len):
    from .deepseek_v3_2.model_args import ModelArgs

    args = ModelArgs()
    cfg = json.loads((Path(model_dir) / "config.json").read_text())
    if cfg.get("num_hidden_layers"):
        args = replace(args, n_layers=int(cfg["num_hidden_layers"]))
    return args if max_seq_len is None else replace(args, max_seq_len=max_seq_len)


def _dsv32_load(model_dir, device, dtype, max_seq_len):
    from tilert_b200.convert import HFCheckpoint

    from .deepseek_v3_2.model import DsaModel

    return DsaModel(_dsv32_args(model_dir, max_seq_len), HFCheckpoint(model_dir), device)


def _dsv32_generator(model_dir, o):
    from tilert_b200.convert import HFCheckpoint

    from .deepseek_v3_2.generator import DSAv32Generator
    from .deepseek_v3_2.model_args import ModelArgs, toy_model_args

    if model_dir is not None:
        margs = _dsv32_args(model_dir, o.max_seq_len)
    elif o.model == "toy":
        margs = replace(toy_model_args(), max_seq_len=o.max_seq_len)
    else:
        margs = replace(ModelArgs(), n_layers=o.layers, n_dense_layers=min(3, o.layers - 1), max_seq_len=o.max_seq_len)
    gen = DSAv32Generator(margs, max_new_tokens=o.max_new_tokens, with_mtp=o.with_mtp, sampling_seed=o.seed, max_seq_len=o.max_seq_len)
    if model_dir is not None:
        ckpt = HFCheckpoint(model_dir)
        gen.from_state_dict({k: ckpt[k] for k in ckpt.keys()})
    else:
        gen.init_random_weights(o.seed)
    return gen


FAMILIES = (
    ModelFamily("deepseek_v3_2", "deepseek_v3_2", ("deepseek_v3_2", "DeepseekV32ForCausalLM", "deepseek_v32"), ("bfloat16",), _dsv32_load, _dsv32_generator,
                presets=("toy", "deepseek_v3_2")),
    ModelFamily("ralasun", "ralasun", ("Ralasun", "ralasun"), ("bfloat16", "float32"), _ralasun_load, _ralasun_generator,
                presets=("ralasun",)),
    ModelFamily("rozesun", "ralasun", ("Rozesun", "rozesun"), ("bfloat16", "float32"), _rozesun_load, _rozesun_generator,
                presets=("rozesun",)),
)


def presets() -> list[str]:
    return [p for f in FAMILIES for p in f.presets]


def family_of_preset(preset: str) -> ModelFamily:
    for f in FAMILIES:
        if preset in f.presets:
            return f
    raise ValueError(f"unknown model {preset!r}; known: {presets()}")


def family_of_dir(model_dir) -> ModelFamily:
    """The family a model directory's ``config.json`` names."""
    cfg = json.loads((Path(model_dir) / "config.json").read_text())
    names = [cfg.get("architecture"), cfg.get("model_type"), *(cfg.get("architectures") or [])]
    for f in FAMILIES:
        if any(n in f.architectures for n in names if n is not None):
            return f
    raise ValueError(f"{model_dir}: no model family for {[n for n in names if n is not None]}; known: "
                     f"{[a for f in FAMILIES for a in f.architectures]}")
