"""Plain, slow restatement of the Ralasun decoder on the CPU -- one function per mechanism, token loops where they
make the rule visible, no code shared with the package.  Everything is computed in the dtype of its inputs
(float64 in the tests that want an exact yardstick).

Notation: x_t is the residual vector of token t, W a weight stored [out, in], n(.) an RMS norm.

    x_t   = n(embed[token_t])
    x_t  += n1(mixer(x)_t)          no norm in front of a sublayer, one behind it
    x_t  += n2(ff(x_t))
    logits_t = head n(x_t)
"""

from __future__ import annotations

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x divided by sqrt(mean(x^2) + eps), over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_around_one(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm whose gain is 1 + w."""
    return rms(x, eps) * (1 + w)


def projection_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm over a whole projection (all heads at once), plain gain."""
    return rms(x, eps) * w


def visible(i: int, size: int | None) -> range:
    """Positions that position i attends to: itself and the size - 1 tokens before it (size None: all)."""
    return range(0 if size is None else max(0, i - size + 1), i + 1)


def mix_values(v: torch.Tensor, first: torch.Tensor, lam: float) -> torch.Tensor:
    """A layer's values pulled towards those of the first mixing layer, position by position."""
    return (1 - lam) * v + lam * first


def attend(q, k, v, heads: int, kv_heads: int, scale: float, size: int | None) -> torch.Tensor:
    """q [T, heads, d], k [T, kv_heads, d], v [T, kv_heads, dv] -> [T, heads, dv]; one query at a time."""
    t = q.shape[0]
    out = torch.zeros(t, heads, v.shape[-1], dtype=q.dtype)
    for i in range(t):
        js = visible(i, size)
        for h in range(heads):
            g = h // (heads // kv_heads)
            s = (k[js.start: js.stop, g] @ q[i, h]) * scale
            out[i, h] = torch.softmax(s, dim=0) @ v[js.start: js.stop, g]
    return out


def gated_unit(gate: torch.Tensor, up: torch.Tensor, limit: float) -> torch.Tensor:
    """Clamped gate and up halves: g sigmoid(1.702 g) (u + 1), g = min(gate, limit), u = up kept in [-limit, limit]."""
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, min=-limit, max=limit)
    return g * (1 / (1 + torch.exp(-1.702 * g))) * (u + 1)


def feed_forward(x, w_gate, w_up, w_down, limit: float) -> torch.Tensor:
    return gated_unit(x @ w_gate.T, x @ w_up.T, limit) @ w_down.T


def route(x: torch.Tensor, w: torch.Tensor, bias: torch.Tensor, top: int) -> tuple[list[int], torch.Tensor]:
    """One token: the `top` experts with the largest logits, and the softmax over those logits alone."""
    z = w @ x + bias
    ids = torch.argsort(z, descending=True, stable=True)[:top].tolist()
    return ids, torch.softmax(z[ids], dim=0)


def route_margin(x: torch.Tensor, w: torch.Tensor, bias: torch.Tensor, top: int) -> float:
    """Distance between the last chosen logit and the first that is not (how close a call the routing is)."""
    z = torch.sort(w @ x + bias, descending=True).values
    return float(z[top - 1] - z[top]) if top < z.numel() else float("inf")


def mixture(x: torch.Tensor, w: dict, p: str, mlp: dict) -> torch.Tensor:
    """Weighted sum of the chosen experts, plus the shared one; token by token."""
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        ids, probs = route(x[t], w[f"{p}.router"], w[f"{p}.router.b"], mlp["router"]["top"])
        for e, pr in zip(ids, probs):
            out[t] += pr * feed_forward(x[t], w[f"{p}.e{e}.gate"], w[f"{p}.e{e}.up"], w[f"{p}.e{e}.down"],
                                        mlp["expert"]["limit"])
        if mlp.get("shared") is not None:
            out[t] += feed_forward(x[t], w[f"{p}.shared.gate"], w[f"{p}.shared.up"], w[f"{p}.shared.down"],
                                   mlp["shared"]["limit"])
    return out


def mixer(x: torch.Tensor, w: dict, p: str, mix: dict, eps: float, first: list) -> torch.Tensor:
    """``first`` is an empty list until the first value-mixing layer puts its values into it."""
    t, h, g, d, dv = x.shape[0], mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = projection_norm(x @ w[f"{p}.q"].T, w[f"{p}.q.norm"], eps).view(t, h, d)
    k = projection_norm(x @ w[f"{p}.k"].T, w[f"{p}.k.norm"], eps).view(t, g, d)
    v = x @ w[f"{p}.v"].T
    if mix.get("v_mix"):
        if not first:
            first.append(v)
        else:
            v = mix_values(v, first[0], float(w[f"{p}.vmix"]))
    size = mix["mask"]["size"] if mix.get("mask") else None
    o = attend(q, k, v.view(t, g, dv), h, g, mix["scale"], size)
    return o.reshape(t, h * dv) @ w[f"{p}.o"].T


def forward(cfg: dict, weights: dict, tokens: list[int], dtype=torch.float64, layers_out: list | None = None,
            margins: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence; ``layers_out`` receives the residual stream after every layer,
    ``margins`` every token's smallest routing margin over the layers."""
    closest = torch.full((len(tokens),), float("inf"))
    w = {k: t.to(dtype) for k, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = norm_around_one(w["embed"][torch.tensor(tokens)], w["embed.norm"], eps)
    first: list = []
    for i, layer in enumerate(cfg["layers"]):
        x = x + norm_around_one(mixer(x, w, f"l{i}.mix", layer["mixer"], eps, first), w[f"l{i}.norm1"], eps)
        if layer.get("mlp") is not None:
            if margins is not None:
                m, top = f"l{i}.mlp", layer["mlp"]["router"]["top"]
                here = [route_margin(r, w[f"{m}.router"], w[f"{m}.router.b"], top) for r in x]
                closest = torch.minimum(closest, torch.tensor(here))
            x = x + norm_around_one(mixture(x, w, f"l{i}.mlp", layer["mlp"]), w[f"l{i}.norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    if margins is not None:
        margins.extend(closest.tolist())
    return norm_around_one(x, w["final.norm"], eps) @ w["head"].T
