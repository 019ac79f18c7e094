"""Differential attention over the paged cache: every head attends with two maps over the same values, and the second
map's output is subtracted from the first's.

A query head has two query parts of ``dim`` elements, a key/value head two key parts and ``value_dim`` values; part c of
a query meets part c of its keys.  With a_1 and a_2 the outputs of the two softmax maps of a head,

    lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff          (one number for the layer)
    o = a_1 - lambda * a_2,   o <- (1 - diff) * o / sqrt(mean(o^2) + eps)

and the output projection follows on the concatenated heads.

How it runs.  The two key parts of a head lie side by side in ONE cached key row of ``2 * dim`` elements beside the
values (no value is cached twice), and a query head becomes two query heads of the attention kernels, [part 1 | 0] and
[0 | part 2] (`ops.heads_to_pages`): their scores with such a row are the two maps' scores, so every paged attention
kernel is used as it is, with an even number of query heads per key/value head.  The prefill kernels form the difference
and its norm in float32 registers as they write; behind the others `ops.diff_combine` does, on float32 outputs."""

from __future__ import annotations

import math

import torch

from slipstream_b200 import ops

from .attention import PagedAttention
from .base import MIXERS, IntoNorm, LayerBinding, PositionEncoding, Runtime, WeightSpec


@MIXERS.register("differential_attention")
class DifferentialAttention(PagedAttention):
    takes_into = True
    takes_pending_norm = True

    def __init__(self, name: str, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int, value_dim: int,
                 position_encoding: PositionEncoding, diff: float, norm_eps: float, *, scale: float | None = None,
                 qkv_bias: bool = True, window: int | None = None, keep_first: int = 0, page_size: int | None = None,
                 names: dict[str, str] | None = None) -> None:
        """``names``: the checkpoint's tensor names by role (q, k, v, o, q_bias, k_bias, v_bias, lq1, lk1, lq2, lk2)."""
        if not 1 <= dim <= 128:
            raise ValueError(f"a map's size is between 1 and 128, not {dim}")
        # to the kernels: two query heads per head, on key rows that hold both parts
        super().__init__(name, hidden_size, 2 * num_heads, num_kv_heads, 2 * dim, position_encoding, qkv_bias=qkv_bias,
                         window=window, scale=dim ** -0.5 if scale is None else scale, page_size=page_size, value_dim=value_dim,
                         keep_first=keep_first, names={**{r: f"{name}.{r}" for r in ("lq1", "lk1", "lq2", "lk2")}, **(names or {})})
        if num_heads % num_kv_heads:
            raise ValueError(f"num_heads ({num_heads}) must be divisible by num_kv_heads ({num_kv_heads})")
        self.heads, self.dim = num_heads, dim
        self.diff, self.norm_eps = float(diff), float(norm_eps)

    @property
    def spread(self) -> bool:
        return True

    def weight_specs(self) -> list[WeightSpec]:
        h, d, names = self.hidden_size, self.dim, self.names
        rows = {"q": self.heads * 2 * d, "k": self.num_kv_heads * 2 * d, "v": self.num_kv_heads * self.value_dim}
        specs = [WeightSpec(names[role], (n, h)) for role, n in rows.items()]
        specs.append(WeightSpec(names["o"], (h, self.heads * self.value_dim)))
        if self.qkv_bias:
            specs += [WeightSpec(names[f"{role}_bias"], (n,), kind="vector") for role, n in rows.items()]
        specs += [WeightSpec(names[role], (d,), kind="vector", init=("normal", 0.1)) for role in ("lq1", "lk1", "lq2", "lk2")]
        return specs

    def bind(self, weights: dict[str, torch.Tensor], runtime: Runtime) -> None:
        self.runtime = runtime
        names, roles = self.names, ("q", "k", "v")
        stacked = [weights[names[r]] for r in roles]
        self.k_col = stacked[0].shape[0]
        self.v_col = self.k_col + stacked[1].shape[0]
        pad = -sum(t.shape[0] for t in stacked) % 8  # rows of 16-byte multiples
        if pad:
            stacked.append(stacked[0].new_zeros((pad, self.hidden_size)))
        self.qkv_weight = torch.cat(stacked).contiguous()
        self.qkv_b = None
        if self.qkv_bias:
            biases = [weights[names[f"{r}_bias"]].to(runtime.dtype) for r in roles]
            self.qkv_b = torch.cat([*biases, biases[0].new_zeros(pad)]).contiguous()
        self.o_weight, self.o_b = weights[names["o"]], None
        lq1, lk1, lq2, lk2 = (weights[names[r]].to(torch.float64).cpu() for r in ("lq1", "lk1", "lq2", "lk2"))
        lam = math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + self.diff
        self.pair = ops.DiffPair(lam, 1.0 - self.diff, self.norm_eps, self.value_dim)
        self.position_encoding.bind(weights, runtime)
        ops.attention_library(self.head_dim)  # compile now, not inside the first step

    def forward(self, x: torch.Tensor, ctx, layer: LayerBinding, into: IntoNorm | None = None) -> torch.Tensor:
        self._check_spread(layer)
        meta = ctx.groups[layer.group]
        rows = ops.linear(x, self.qkv_weight, self.qkv_b)
        inv_freq, rotary_dim = self.position_encoding.rotary_table()
        q = ops.heads_to_pages(rows, ctx.positions, meta.slot_mapping, layer.kv, self.heads, self.num_kv_heads, self.dim,
                               self.value_dim, self.head_dim, self.k_col, self.v_col, maps=2, inv_freq=inv_freq,
                               rotary_dim=rotary_dim, interleaved=getattr(self.position_encoding, "interleaved", False))
        out = torch.empty((x.shape[0], self.heads * self.value_dim), dtype=q.dtype, device=q.device)
        ops.paged_attention(q, out, layer.kv, meta.block_tables, ctx, self.num_heads, self.num_kv_heads, self.head_dim,
                            self.scale, self.window or 0, keep=self.keep_first, diff=self.pair)
        if into is not None:
            return into.close(out, self.o_weight, self.o_b)
        return ops.linear(out, self.o_weight, self.o_b)
