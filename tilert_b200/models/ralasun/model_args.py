"""Configuration of a Ralasun decoder: every size and constant is per layer and comes from ``config.json``."""

from __future__ import annotations

import json
from dataclasses import dataclass, replace
from pathlib import Path

GATE_ALPHA = 1.702  # slope of the sigmoid in the experts' gated unit


@dataclass(frozen=True)
class MixerArgs:
    heads: int
    kv_heads: int
    dim: int               # query / key size per head
    vdim: int              # value size per head
    window: int | None     # positions a query sees, itself included (None: all before it)
    scale: float           # factor on q . k
    v_mix: bool            # values are mixed with those of the first layer that has this set


@dataclass(frozen=True)
class MlpArgs:
    experts: int
    top: int
    ff: int
    limit: float
    shared_ff: int = 0     # 0: no shared expert
    shared_limit: float = 0.0


@dataclass(frozen=True)
class LayerArgs:
    mixer: MixerArgs
    mlp: MlpArgs | None    # None: the layer has no feed-forward


@dataclass(frozen=True)
class RalasunArgs:
    vocab_size: int
    dim: int
    eps: float
    layers: tuple[LayerArgs, ...]
    max_seq_len: int = 4096
    arch_name: str = "ralasun"

    def __post_init__(self):
        first = None
        for i, layer in enumerate(self.layers):
            m, f = layer.mixer, layer.mlp
            if m.heads % m.kv_heads != 0:
                raise ValueError(f"layer {i}: {m.heads} query heads do not divide over {m.kv_heads} key/value heads")
            if m.window is not None and m.window < 1:
                raise ValueError(f"layer {i}: window {m.window}")
            if f is not None and not 1 <= f.top <= f.experts:
                raise ValueError(f"layer {i}: {f.top} of {f.experts} experts per token")
            if m.v_mix:
                n = m.kv_heads * m.vdim
                first = n if first is None else first
                if n != first:
                    raise ValueError(f"layer {i}: {n} value rows, but the first value-mixing layer has {first}")

    @classmethod
    def from_config(cls, cfg: dict, max_seq_len: int | None = None) -> "RalasunArgs":
        layers = []
        for i, entry in enumerate(cfg["layers"]):
            if entry["type"] != "attention":
                raise ValueError(f"layer {i}: unknown mixer type {entry['type']!r}")
            m = entry["mixer"]
            mask = m.get("mask")
            mixer = MixerArgs(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                              window=None if mask is None else int(mask["size"]), scale=float(m["scale"]),
                              v_mix=bool(m.get("v_mix", False)))
            f = entry.get("mlp")
            mlp = None
            if f is not None:
                if f["kind"] != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
                sh = f.get("shared")
                mlp = MlpArgs(experts=int(f["router"]["experts"]), top=int(f["router"]["top"]), ff=int(f["expert"]["ff"]),
                              limit=float(f["expert"]["limit"]), shared_ff=0 if sh is None else int(sh["ff"]),
                              shared_limit=0.0 if sh is None else float(sh["limit"]))
            layers.append(LayerArgs(mixer, mlp))
        args = cls(vocab_size=int(cfg["vocab"]), dim=int(cfg["width"]), eps=float(cfg["norm"]["eps"]), layers=tuple(layers))
        return args if max_seq_len is None else replace(args, max_seq_len=max_seq_len)

    @classmethod
    def from_dir(cls, model_dir, max_seq_len: int | None = None) -> "RalasunArgs":
        return cls.from_config(json.loads((Path(model_dir) / "config.json").read_text()), max_seq_len)

    def to_config(self) -> dict:
        """The ``config.json`` that ``from_config`` reads back."""
        layers = []
        for layer in self.layers:
            m, f = layer.mixer, layer.mlp
            mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "v_mix": m.v_mix,
                     "mask": None if m.window is None else {"size": m.window}}
            mlp = None
            if f is not None:
                mlp = {"kind": "moe", "router": {"experts": f.experts, "top": f.top}, "expert": {"ff": f.ff, "limit": f.limit},
                       "shared": {"ff": f.shared_ff, "limit": f.shared_limit} if f.shared_ff else None}
            layers.append({"type": "attention", "mixer": mixer, "mlp": mlp})
        return {"architecture": "Ralasun", "vocab": self.vocab_size, "width": self.dim, "norm": {"eps": self.eps}, "layers": layers}


def uniform_args(n_layers: int, dim: int, vocab: int, mixer: MixerArgs, mlp: MlpArgs | None, eps: float = 1e-6,
                 max_seq_len: int = 4096) -> RalasunArgs:
    """A model whose layers are all alike."""
    return RalasunArgs(vocab, dim, eps, (LayerArgs(mixer, mlp),) * n_layers, max_seq_len)


def toy_args(max_seq_len: int = 1024) -> RalasunArgs:
    """A small random-weight model for the command line and the tests: unequal layers, one of them without a
    feed-forward, one outside the value mixing."""
    def mixer(window, v_mix=True, heads=6, dim=40):
        return MixerArgs(heads=heads, kv_heads=2, dim=dim, vdim=48, window=window, scale=dim ** -0.5, v_mix=v_mix)

    mlp = MlpArgs(experts=10, top=3, ff=72, limit=1.5, shared_ff=104, shared_limit=2.5)
    return RalasunArgs(vocab_size=768, dim=256, eps=1e-6, max_seq_len=max_seq_len, layers=(
        LayerArgs(mixer(33), mlp), LayerArgs(mixer(50, v_mix=False, heads=4, dim=64), None), LayerArgs(mixer(20), mlp)))
