"""A plain, slow implementation of the Sazepel decoder in double precision on the CPU: one function per mechanism,
written from the design's equations, sharing no code with the package.  Tests compare the engine with it.

``config`` is the design's nested dictionary (what its config.json holds), ``weights`` a dictionary from tensor name
to a float64 tensor.  A whole sequence is run at once: ``forward(config, weights, tokens)`` returns the logits of
every position and, on request, the residual stream after every layer.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """Divided by its root mean square over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm(x: torch.Tensor, g: torch.Tensor, eps: float) -> torch.Tensor:
    """``g``: one number for all coordinates, or one per coordinate."""
    return unit(x, eps) * g


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def rotate(x: torch.Tensor, rot: dict | None) -> torch.Tensor:
    """``x`` [T, heads, D]: elements i and i + dims/2 of every head turned by position * base^(-2i/dims)."""
    if not rot:
        return x
    t, dims = x.shape[0], rot["dims"]
    half = dims // 2
    freq = rot["base"] ** (-2.0 * torch.arange(half, dtype=F64) / dims)
    angle = torch.arange(t, dtype=F64)[:, None] * freq[None, :]
    cos, sin = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    out = x.clone()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * cos - v * sin
    out[..., half:dims] = v * cos + u * sin
    return out


# --------------------------------------------------------------------------- mixers

def retention_heads(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: list) -> torch.Tensor:
    """Token by token: S <- decay S + k v^T, o = S^T q per head.  [T, heads, ...] -> [T, heads, vdim]."""
    t, heads, d = q.shape
    state = torch.zeros(heads, d, v.shape[2], dtype=F64)
    dec = torch.tensor(decay, dtype=F64)[:, None, None]
    out = []
    for i in range(t):
        state = dec * state + k[i][:, :, None] * v[i][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", state, q[i]))
    return torch.stack(out)


def retention(m: dict, w: dict, p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    t, heads, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = rotate((h @ w[f"{p}.q"].T).reshape(t, heads, d), m.get("rot"))
    k = rotate((h @ w[f"{p}.k"].T).reshape(t, heads, d), m.get("rot")) * d ** -0.5
    v = (h @ w[f"{p}.v"].T).reshape(t, heads, dv)
    o = unit(retention_heads(q, k, v, m["decay"]), eps).reshape(t, heads * dv)
    return (o * silu(h @ w[f"{p}.g"].T)) @ w[f"{p}.o"].T


def head_weights(q: torch.Tensor, k: torch.Tensor, scale: float) -> torch.Tensor:
    """Causal softmax weights of every head, [H, T, T]; q [T, H, d], k [T, G, d]."""
    t, heads = q.shape[:2]
    k = k.repeat_interleave(heads // k.shape[1], dim=1)
    scores = torch.einsum("ihd,jhd->hij", q, k) * scale
    return torch.softmax(scores.masked_fill(~torch.tril(torch.ones(t, t, dtype=torch.bool)), -math.inf), dim=-1)


def talk(weights: torch.Tensor, table: torch.Tensor) -> torch.Tensor:
    """Head h's weights become sum_g table[h, g] weights_g."""
    return torch.einsum("hg,gij->hij", table, weights)


def talking_attention(m: dict, w: dict, p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    t, heads, groups, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit((h @ w[f"{p}.q"].T).reshape(t, heads, d), eps)
    k = unit((h @ w[f"{p}.k"].T).reshape(t, groups, d), eps)
    v = unit((h @ w[f"{p}.v"].T).reshape(t, groups, dv), eps)
    mixed = talk(head_weights(q, k, m["scale"]), w[f"{p}.talk"])
    o = torch.einsum("hij,jhv->ihv", mixed, v.repeat_interleave(heads // groups, dim=1)).reshape(t, heads * dv)
    return (o * torch.sigmoid(h @ w[f"{p}.g"].T)) @ w[f"{p}.o"].T


def parallel(m: dict, w: dict, p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    left = talking_attention(m["left"], w, f"{p}.left", h, eps)
    right = retention(m["right"], w, f"{p}.right", h, eps)
    return 0.5 * (norm(left, w[f"{p}.left.out"], eps) + norm(right, w[f"{p}.right.out"], eps))


# --------------------------------------------------------------------------- feed-forward

def expert(w: dict, p: str, h: torch.Tensor) -> torch.Tensor:
    return (silu(h @ w[f"{p}.gate"].T) * (h @ w[f"{p}.up"].T)) @ w[f"{p}.down"].T


def route(mlp: dict, w: dict, p: str, h: torch.Tensor) -> tuple[torch.Tensor, torch.Tensor]:
    """(chosen experts [T, top], their weights [T, top])."""
    z = h @ w[f"{p}.router"].T + w[f"{p}.router.b"]
    best = z.topk(mlp["router"]["top"], dim=-1)
    return best.indices, torch.softmax(best.values, dim=-1)


def routed_experts(mlp: dict, w: dict, p: str, h: torch.Tensor) -> torch.Tensor:
    ids, weights = route(mlp, w, p, h)
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, places = (ids == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += weights[rows, places][:, None] * expert(w, f"{p}.e{e}", h[rows])
    return out


# --------------------------------------------------------------------------- the model

def forward(config: dict, weights: dict, tokens: list[int], want_layers: bool = False):
    eps, w = config["norm"]["eps"], weights
    x = norm(w["embed"][torch.tensor(tokens)], w["embed.norm"], eps)
    layers = []
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}", layer["mixer"]
        h = norm(x, w[f"{p}.norm1"], eps)
        mixer = {"retention": retention, "parallel": parallel}[layer["type"]]
        x = x + norm(mixer(m, w, f"{p}.mix", h, eps), w[f"{p}.norm1b"], eps)
        if layer.get("mlp"):
            y = routed_experts(layer["mlp"], w, f"{p}.mlp", norm(x, w[f"{p}.norm2"], eps))
            x = x + norm(y, w[f"{p}.norm2b"], eps)
        layers.append(x)
    logits = norm(x, w["final.norm"], eps) @ w["head"].T * config.get("logit_scale", 1.0)
    return (logits, torch.stack(layers)) if want_layers else logits
