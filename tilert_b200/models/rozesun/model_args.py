"""Configuration of a Rozesun decoder: every size and constant is per layer and comes from ``config.json``; what its two
kinds of mixer have is fixed by the design."""

from __future__ import annotations

import json
from dataclasses import dataclass, replace
from pathlib import Path

GATE_ALPHA = 1.702  # slope of the sigmoid in the feed-forward's gated unit


@dataclass(frozen=True)
class MixerKind:
    interleaved: bool      # rotated pairs are neighbours (else: halves apart)
    windowed: bool         # a query sees the last positions only
    sink: bool             # a learned term in the softmax denominator, per head
    gate_per_head: bool    # the output gate has one value per head (else: one per element)


KINDS = {
    "latent_attention": MixerKind(interleaved=False, windowed=False, sink=False, gate_per_head=False),
    "latent_attention_2": MixerKind(interleaved=True, windowed=True, sink=True, gate_per_head=True),
}


@dataclass(frozen=True)
class MixerArgs:
    kind: str              # a key of KINDS
    heads: int
    dim: int               # query / key size per head that is not rotated
    rot_dim: int           # query / key size that is
    vdim: int              # value size per head
    q_rank: int            # size of the queries' latent
    kv_rank: int           # size of the keys' and values' latent
    scale: float           # factor on q . k
    rot_base: float
    window: int | None = None  # positions a query sees, itself included (None: all before it)

    @property
    def interleaved(self) -> bool:
        return KINDS[self.kind].interleaved

    @property
    def sink(self) -> bool:
        return KINDS[self.kind].sink

    @property
    def gate_per_head(self) -> bool:
        return KINDS[self.kind].gate_per_head

    @property
    def gate_rows(self) -> int:
        return self.heads if self.gate_per_head else self.heads * self.vdim


@dataclass(frozen=True)
class MlpArgs:
    ff: int
    limit: float


@dataclass(frozen=True)
class LayerArgs:
    mixer: MixerArgs
    mlp: MlpArgs | None    # None: the layer has no feed-forward


@dataclass(frozen=True)
class LoopArgs:
    """Layers start .. stop - 1 run ``times`` times in a row, each pass with caches of its own."""

    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class RozesunArgs:
    vocab_size: int
    dim: int
    eps: float
    logit_scale: float
    layers: tuple[LayerArgs, ...]
    loop: LoopArgs | None = None
    max_seq_len: int = 4096
    arch_name: str = "rozesun"

    def __post_init__(self):
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            if m.kind not in KINDS:
                raise ValueError(f"layer {i}: unknown mixer type {m.kind!r}")
            if KINDS[m.kind].windowed != (m.window is not None):
                raise ValueError(f"layer {i}: a mixer of type {m.kind} {'needs a' if m.window is None else 'has no'} window")
            if m.window is not None and m.window < 1:
                raise ValueError(f"layer {i}: window {m.window}")
            if m.rot_dim < 2 or m.rot_dim % 2 != 0:
                raise ValueError(f"layer {i}: {m.rot_dim} rotated dimensions do not pair up")
        lp = self.loop
        if lp is not None and not (0 <= lp.start < lp.stop <= len(self.layers) and lp.times >= 1):
            raise ValueError(f"loop over layers {lp.start} .. {lp.stop - 1}, {lp.times} times: there are {len(self.layers)} layers")

    def runs(self) -> list[tuple[int, int | None]]:
        """(layer, number of the pass that begins with it or None) in the order of computation."""
        n, lp = len(self.layers), self.loop
        if lp is None:
            return [(i, None) for i in range(n)]
        out: list[tuple[int, int | None]] = [(i, None) for i in range(lp.start)]
        for t in range(lp.times):
            out += [(i, t if i == lp.start else None) for i in range(lp.start, lp.stop)]
        return out + [(i, None) for i in range(lp.stop, n)]

    @classmethod
    def from_config(cls, cfg: dict, max_seq_len: int | None = None) -> "RozesunArgs":
        layers = []
        for i, entry in enumerate(cfg["layers"]):
            m = entry["mixer"]
            if int(m["rot"]["dims"]) != int(m["rot_dim"]):
                raise ValueError(f"layer {i}: {m['rot']['dims']} of {m['rot_dim']} dimensions rotated")
            mask = m.get("mask")
            mixer = MixerArgs(kind=entry["type"], heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                              q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), rot_base=float(m["rot"]["base"]),
                              window=None if mask is None else int(mask["size"]))
            f = entry.get("mlp")
            if f is not None and f["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
            layers.append(LayerArgs(mixer, None if f is None else MlpArgs(int(f["ff"]), float(f["limit"]))))
        lp = cfg.get("loop")
        args = cls(vocab_size=int(cfg["vocab"]), dim=int(cfg["width"]), eps=float(cfg["norm"]["eps"]), logit_scale=float(cfg["logit_scale"]),
                   layers=tuple(layers), loop=None if lp is None else LoopArgs(int(lp["start"]), int(lp["stop"]), int(lp["times"])))
        return args if max_seq_len is None else replace(args, max_seq_len=max_seq_len)

    @classmethod
    def from_dir(cls, model_dir, max_seq_len: int | None = None) -> "RozesunArgs":
        return cls.from_config(json.loads((Path(model_dir) / "config.json").read_text()), max_seq_len)

    def to_config(self) -> dict:
        """The ``config.json`` that ``from_config`` reads back."""
        layers = []
        for layer in self.layers:
            m, f = layer.mixer, layer.mlp
            mixer = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "q_rank": m.q_rank, "kv_rank": m.kv_rank,
                     "scale": m.scale, "rot": {"base": m.rot_base, "dims": m.rot_dim}}
            if m.window is not None:
                mixer["mask"] = {"size": m.window}
            layers.append({"type": m.kind, "mixer": mixer, "mlp": None if f is None else {"kind": "dense", "ff": f.ff, "limit": f.limit}})
        lp = self.loop
        return {"architecture": "Rozesun", "vocab": self.vocab_size, "width": self.dim, "norm": {"eps": self.eps},
                "logit_scale": self.logit_scale, "layers": layers,
                "loop": None if lp is None else {"start": lp.start, "stop": lp.stop, "times": lp.times}}


def uniform_args(n_layers: int, dim: int, vocab: int, mixer: MixerArgs, mlp: MlpArgs | None, eps: float = 1e-6,
                 max_seq_len: int = 4096) -> RozesunArgs:
    """A model whose layers are all alike, none of them looped."""
    return RozesunArgs(vocab, dim, eps, 1.0, (LayerArgs(mixer, mlp),) * n_layers, None, max_seq_len)


def toy_args(max_seq_len: int = 1024) -> RozesunArgs:
    """A small random-weight model for the command line and the tests: both kinds of mixer, unequal sizes, a loop over
    the two middle layers, a layer without a feed-forward."""
    wide = MixerArgs("latent_attention", heads=6, dim=40, rot_dim=24, vdim=48, q_rank=56, kv_rank=72, scale=0.125, rot_base=9000.0)
    near = MixerArgs("latent_attention_2", heads=5, dim=48, rot_dim=16, vdim=32, q_rank=64, kv_rank=48, scale=0.11, rot_base=700.0, window=33)
    return RozesunArgs(vocab_size=768, dim=192, eps=1e-6, logit_scale=0.4, max_seq_len=max_seq_len, loop=LoopArgs(1, 3, 2), layers=(
        LayerArgs(near, MlpArgs(296, 1.5)), LayerArgs(wide, MlpArgs(320, 2.0)), LayerArgs(near, None), LayerArgs(wide, MlpArgs(296, 1.5))))
