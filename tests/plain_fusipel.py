"""A plain, slow implementation of the Fusipel decoder in double precision on the CPU: one function per mechanism,
written from the design's equations, sharing no code with the package.  Tests compare the engine with it.

``config`` is the design's nested dictionary (what its config.json holds), ``weights`` a dictionary from tensor name
to a float64 tensor.  A whole sequence is run at once: ``forward(config, weights, tokens)`` returns the logits of
every position and, on request, the residual stream after every layer run.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms(x, eps) * w


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# --------------------------------------------------------------------------- positions

def frequencies(rot: dict) -> torch.Tensor:
    """One frequency per pair; waves longer than the trained context turn ``factor`` times slower, those short enough
    as before, those between by a blend of the two."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        s = rot.get("scaling")
        if s:
            wave = 2.0 * math.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wave >= s["original"] / s["high"]:
                t = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - t) * f / s["factor"] + t * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate(x: torch.Tensor, rot: dict | None) -> torch.Tensor:
    """``x`` [T, ..., D]: neighbours (2i, 2i + 1) of the first ``dims`` elements turned by position * frequency i."""
    if not rot:
        return x
    t, dims = x.shape[0], rot["dims"]
    angle = torch.arange(t, dtype=F64)[:, None] * frequencies(rot)[None, :]
    angle = angle.reshape(t, *([1] * (x.dim() - 2)), dims // 2)
    cos, sin = torch.cos(angle), torch.sin(angle)
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def visible(t: int, mask: dict | None) -> torch.Tensor:
    i, j = torch.arange(t)[:, None], torch.arange(t)[None, :]
    seen = j <= i
    if mask:
        seen = seen & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))
    return seen


# --------------------------------------------------------------------------- mixers

def differential_lambda(w: dict, p: str, diff: float) -> float:
    return float(torch.exp((w[f"{p}.lq1"] * w[f"{p}.lk1"]).sum()) - torch.exp((w[f"{p}.lq2"] * w[f"{p}.lk2"]).sum())) + diff


def differential_combine(a1: torch.Tensor, a2: torch.Tensor, lam: float, diff: float, eps: float) -> torch.Tensor:
    """Heads' outputs of the two maps [..., vdim] into one: a difference, over its root mean square, times 1 - diff."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def differential_attention(m: dict, w: dict, p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    t, heads, groups, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate((h @ w[f"{p}.q"].T + w[f"{p}.q.b"]).reshape(t, heads, 2, d), m.get("rot"))
    k = rotate((h @ w[f"{p}.k"].T + w[f"{p}.k.b"]).reshape(t, groups, 2, d), m.get("rot"))
    v = (h @ w[f"{p}.v"].T + w[f"{p}.v.b"]).reshape(t, groups, dv)
    seen = visible(t, m.get("mask"))
    lam = differential_lambda(w, p, m["diff"])
    out = torch.zeros(t, heads, dv, dtype=F64)
    for head in range(heads):
        g = head // (heads // groups)
        maps = []
        for c in range(2):
            scores = (q[:, head, c] @ k[:, g, c].T) * m["scale"]
            maps.append(torch.softmax(scores.masked_fill(~seen, -math.inf), dim=-1) @ v[:, g])
        out[:, head] = differential_combine(maps[0], maps[1], lam, m["diff"], eps)
    return out.reshape(t, heads * dv) @ w[f"{p}.o"].T


def sink_softmax(scores: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """Softmax over the last axis whose denominator also holds exp(sink)."""
    top = torch.maximum(scores.max(dim=-1, keepdim=True).values, sink)
    e = torch.exp(scores - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink - top))


def shared_key_value_attention(m: dict, w: dict, p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    """The values are the keys as projected; queries and keys pass one norm over all heads together."""
    t, heads, groups, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = h @ w[f"{p}.q"].T + w[f"{p}.q.b"]
    k = h @ w[f"{p}.k"].T + w[f"{p}.k.b"]
    v = k.reshape(t, groups, d)
    q = rotate(norm(q, w[f"{p}.q.norm"], eps).reshape(t, heads, d), m.get("rot"))
    k = rotate(norm(k, w[f"{p}.k.norm"], eps).reshape(t, groups, d), m.get("rot"))
    seen = visible(t, None)
    out = torch.zeros(t, heads, d, dtype=F64)
    for head in range(heads):
        g = head // (heads // groups)
        scores = ((q[:, head] @ k[:, g].T) * m["scale"]).masked_fill(~seen, -math.inf)
        out[:, head] = sink_softmax(scores, w[f"{p}.sink"][head]) @ v[:, g]
    return out.reshape(t, heads * d) @ w[f"{p}.o"].T


# --------------------------------------------------------------------------- feed-forward

def dense(w: dict, p: str, h: torch.Tensor) -> torch.Tensor:
    return (gelu_tanh(h @ w[f"{p}.gate"].T) * (h @ w[f"{p}.up"].T)) @ w[f"{p}.down"].T


# --------------------------------------------------------------------------- the model

def layer_runs(config: dict) -> list[tuple[int, bool]]:
    """(layer, does the embedding output join the stream right before it) in running order."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    runs = [(i, False) for i in range(loop["start"])]
    for turn in range(loop["times"]):
        runs += [(i, turn > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, False) for i in range(loop["stop"], n)]


def forward(config: dict, weights: dict, tokens: list[int], want_layers: bool = False):
    eps, scale, w = config["norm"]["eps"], config["residual_mult"], weights
    x = embedded = w["embed"][torch.tensor(tokens)]
    layers = []
    for i, joins in layer_runs(config):
        layer, p = config["layers"][i], f"l{i}"
        if joins:
            x = x + embedded
        h = norm(x, w[f"{p}.norm1"], eps)
        mixer = {"attention": differential_attention, "attention_2": shared_key_value_attention}[layer["type"]]
        x = x + scale * norm(mixer(layer["mixer"], w, f"{p}.mix", h, eps), w[f"{p}.norm1b"], eps)
        if layer.get("mlp"):
            h = norm(x, w[f"{p}.norm2"], eps)
            x = x + scale * norm(dense(w, f"{p}.mlp", h), w[f"{p}.norm2b"], eps)
        layers.append(x)
    logits = norm(x, w["final.norm"], eps) @ w["head"].T
    return (logits, torch.stack(layers)) if want_layers else logits
