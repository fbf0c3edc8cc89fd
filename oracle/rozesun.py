"""Plain, slow restatement of the Rozesun decoder on the CPU -- one function per mechanism, token loops where they make
the rule visible, no code shared with the package.  Everything is computed in the dtype of its inputs (float64 in the
tests that want an exact yardstick).

Notation: x_t is the residual vector of token t, W a weight stored [out, in], N(.) a layer norm, n(.) an RMS norm.

    x_t   = embed[token_t]
    x_t  += step[r]                          only in front of pass r of the looped block of layers
    x_t  += N1b(mixer(N1(x))_t)
    x_t  += N2b(ff(N2(x))_t)
    logits_t = s * embed N(x_t)
"""

from __future__ import annotations

import torch

from .ralasun import feed_forward, projection_norm, visible


def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    """Mean taken off, divided by the root of (mean squared deviation + eps), times w, plus b."""
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w + b


def rotate(v: torch.Tensor, pos: int, base: float, dims: int, interleaved: bool) -> torch.Tensor:
    """v [.., d] at position `pos`: pair i of the first `dims` elements turns by pos * base^(-2i / dims).  Pair i is
    (2i, 2i + 1) when interleaved, (i, i + dims / 2) otherwise."""
    out = v.clone()
    for i in range(dims // 2):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
        angle = torch.tensor(float(pos) * base ** (-2.0 * i / dims), dtype=torch.float64)
        c, s = torch.cos(angle).to(v.dtype), torch.sin(angle).to(v.dtype)
        out[..., a] = v[..., a] * c - v[..., b] * s
        out[..., b] = v[..., b] * c + v[..., a] * s
    return out


def sink_softmax(s: torch.Tensor, sink: torch.Tensor | None) -> torch.Tensor:
    """Softmax of the scores s; with a sink the denominator has one more term, exp(sink), and the weights sum to less
    than one."""
    if sink is None:
        return torch.softmax(s, dim=-1)
    return torch.softmax(torch.cat([s, sink.reshape(1)]), dim=-1)[:-1]


def latent_keys(h: torch.Tensor, w: dict, p: str, mix: dict, eps: float, interleaved: bool):
    """What a token leaves behind for later ones: the normed latent [T, kv_rank] and the turned key part [T, rot_dim]."""
    r = mix["kv_rank"]
    z = h @ w[f"{p}.dkv"].T
    c = projection_norm(z[:, :r], w[f"{p}.dkv.norm"], eps)
    kr = torch.stack([rotate(z[t, r:], t, mix["rot"]["base"], mix["rot"]["dims"], interleaved) for t in range(h.shape[0])])
    return c, kr


def latent_queries(h: torch.Tensor, w: dict, p: str, mix: dict, eps: float, interleaved: bool):
    """(unturned part [T, H, dim], turned part [T, H, rot_dim])."""
    t, nh, d, r = h.shape[0], mix["heads"], mix["dim"], mix["rot_dim"]
    cq = projection_norm(h @ w[f"{p}.dq"].T, w[f"{p}.dq.norm"], eps)
    q = (cq @ w[f"{p}.uq"].T).view(t, nh, d + r)
    qr = torch.stack([rotate(q[i, :, d:], i, mix["rot"]["base"], mix["rot"]["dims"], interleaved) for i in range(t)])
    return q[:, :, :d], qr


def latent_attend(qn, qr, c, kr, w_uk, w_uv, scale: float, size: int | None, sink=None) -> torch.Tensor:
    """Keys and values are expanded from the latent head by head; one query at a time -> [T, H, vdim]."""
    t, nh, d = qn.shape
    vd = w_uv.shape[0] // nh
    out = torch.zeros(t, nh, vd, dtype=qn.dtype)
    k = (c @ w_uk.T).view(t, nh, d)
    v = (c @ w_uv.T).view(t, nh, vd)
    for i in range(t):
        js = visible(i, size)
        for h in range(nh):
            s = (k[js.start: js.stop, h] @ qn[i, h] + kr[js.start: js.stop] @ qr[i, h]) * scale
            out[i, h] = sink_softmax(s, None if sink is None else sink[h]) @ v[js.start: js.stop, h]
    return out


def gate(o: torch.Tensor, z: torch.Tensor) -> torch.Tensor:
    """o [T, H, vdim] times sigmoid(z), z [T, H * vdim] (every element) or [T, H] (every head) -> [T, H * vdim]."""
    t, nh, vd = o.shape
    g = 1 / (1 + torch.exp(-z))
    g = g.view(t, nh, -1)  # one column or vdim of them
    return (o * g).reshape(t, nh * vd)


# What the two kinds of mixer have: pairs of the rotation, a window, a sink.  (The gate's form follows from its tensor.)
KINDS = {"latent_attention": dict(interleaved=False, window=False, sink=False),
         "latent_attention_2": dict(interleaved=True, window=True, sink=True)}


def mixer(h: torch.Tensor, w: dict, p: str, kind: str, mix: dict, eps: float) -> torch.Tensor:
    k = KINDS[kind]
    c, kr = latent_keys(h, w, p, mix, eps, k["interleaved"])
    qn, qr = latent_queries(h, w, p, mix, eps, k["interleaved"])
    o = latent_attend(qn, qr, c, kr, w[f"{p}.uk"], w[f"{p}.uv"], mix["scale"], mix["mask"]["size"] if k["window"] else None,
                      w[f"{p}.sink"] if k["sink"] else None)
    return gate(o, h @ w[f"{p}.g"].T) @ w[f"{p}.o"].T


def runs(n_layers: int, loop: dict | None) -> list[tuple[int, int | None]]:
    """(layer, pass that begins here or None) in the order of computation."""
    if loop is None:
        return [(i, None) for i in range(n_layers)]
    body = range(loop["start"], loop["stop"])
    out: list[tuple[int, int | None]] = [(i, None) for i in range(loop["start"])]
    for r in range(loop["times"]):
        out += [(i, r if i == loop["start"] else None) for i in body]
    return out + [(i, None) for i in range(loop["stop"], n_layers)]


def forward(cfg: dict, weights: dict, tokens: list[int], dtype=torch.float64, layers_out: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence; ``layers_out`` receives the residual stream after every layer run."""
    w = {k: t.to(dtype) for k, t in weights.items()}
    eps = cfg["norm"]["eps"]

    def norm(x, name):
        return layer_norm(x, w[name], w[f"{name}.b"], eps)

    x = w["embed"][torch.tensor(tokens)]
    for i, begins in runs(len(cfg["layers"]), cfg.get("loop")):
        layer = cfg["layers"][i]
        if begins is not None:
            x = x + w["loop.step"][begins]
        x = x + norm(mixer(norm(x, f"l{i}.norm1"), w, f"l{i}.mix", layer["type"], layer["mixer"], eps), f"l{i}.norm1b")
        if layer.get("mlp") is not None:
            m = f"l{i}.mlp"
            y = feed_forward(norm(x, f"l{i}.norm2"), w[f"{m}.gate"], w[f"{m}.up"], w[f"{m}.down"], layer["mlp"]["limit"])
            x = x + norm(y, f"l{i}.norm2b")
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, "final.norm") @ w["embed"].T * cfg["logit_scale"]
