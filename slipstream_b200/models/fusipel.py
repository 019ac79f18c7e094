"""Builder of the Fusipel decoder from ``FusipelConfig``: which parts stand in which layer, with which constants and
tensor names.

Embedding ``embed``.  Per layer ``l<i>`` a `SandwichBlock`: a norm in front of and behind each branch
(``l<i>.norm1``, ``l<i>.norm1b``, ``l<i>.norm2``, ``l<i>.norm2b``) and a multiplier on what joins the stream.  The mixer,
by ``type``:

* ``attention``: a `DifferentialAttention` (``l<i>.mix.{q,k,v}`` with biases ``.b``, ``l<i>.mix.{lq1,lk1,lq2,lk2,o}``),
  optionally under a sliding window that keeps the first keys in sight;
* ``attention_2``: a `PagedAttention` with ``tied_values``, a joint norm (``l<i>.mix.{q,k}`` with biases ``.b`` and norms
  ``.norm``) and learned sinks (``l<i>.mix.sink``), ``l<i>.mix.o``;

both with rotary pairs of neighbours, their frequencies stretched by bands when ``rot.scaling`` is given.  The
feed-forward, unless ``mlp`` is null: a `GatedFeedForward` with the tanh form of GELU (``l<i>.mlp.{gate,up,down}``).
``final.norm``, ``head``.

The layers of ``loop`` stand in the model's order once per pass (each pass with pages of its own); the first of every
pass but the first is an entry in front of which the embedding output joins the stream.
"""

from __future__ import annotations

from slipstream_b200.config.fusipel_config import BandedRotaryConfig, FusipelConfig
from slipstream_b200.parts import (GELU_TANH, BandedRotaryEncoding, DifferentialAttention, GatedFeedForward, JoiningNorm,
                                   LMHead, NoPositionEncoding, PagedAttention, RotaryEncoding, SandwichBlock,
                                   TokenEmbedding)

from .decoder import DecoderLM, ExecEntry


def _rotary(rot: BandedRotaryConfig | None, dim: int, made: dict):
    """One encoding object per distinct rotation (layers that rotate alike share the table)."""
    key = (rot, dim)
    if key not in made:
        if rot is None:
            made[key] = NoPositionEncoding()
        elif rot.scaling is None:
            made[key] = RotaryEncoding(dim, rot.base, rot.dims, interleaved=True, exact_table=True)
        else:
            factor, low, high, original = rot.scaling
            made[key] = BandedRotaryEncoding(dim, rot.base, rot.dims, interleaved=True, factor=factor, original=original,
                                             low=low, high=high)
    return made[key]


def build_fusipel(config: FusipelConfig) -> DecoderLM:
    c = config
    width = c.hidden_size
    blocks, rotaries = [], {}

    def norm(tensor: str) -> JoiningNorm:
        return JoiningNorm(tensor, width, c.norm_eps)

    for i, layer in enumerate(c.layers):
        p, m = f"l{i}", layer.mixer
        names = {**{role: f"{p}.mix.{role}" for role in "qkvo"}, **{f"{role}_bias": f"{p}.mix.{role}.b" for role in "qkv"},
                 **{f"{role}_norm": f"{p}.mix.{role}.norm" for role in "qk"}}
        if layer.type == "attention":
            mixer = DifferentialAttention(f"{p}.mix", width, m.heads, m.kv_heads, m.dim, m.vdim, _rotary(m.rot, m.dim, rotaries),
                                          m.diff, c.norm_eps, scale=m.scale, window=m.window, keep_first=m.keep_first, names=names)
        else:
            mixer = PagedAttention(f"{p}.mix", width, m.heads, m.kv_heads, m.dim, _rotary(m.rot, m.dim, rotaries), scale=m.scale,
                                   joint_norm_eps=c.norm_eps, tied_values=True, learned_sinks=True, names=names)
        ffn = None
        if layer.ff is not None:
            ffn = GatedFeedForward(f"{p}.mlp", width, layer.ff, names={role: f"{p}.mlp.{role}" for role in ("gate", "up", "down")},
                                   **GELU_TANH)
        blocks.append(SandwichBlock(mixer, ffn, norm(f"{p}.norm1"), norm(f"{p}.norm1b"),
                                    norm(f"{p}.norm2") if ffn is not None else None,
                                    norm(f"{p}.norm2b") if ffn is not None else None, c.residual_mult))
    return DecoderLM(
        c,
        TokenEmbedding("embed", c.vocab_size, width, tensor="embed"),
        blocks,
        norm("final.norm"),
        LMHead("head", c.vocab_size, width, tied_to=None, tensor="head"),
        order=[ExecEntry(i, add_embedding=joins) for i, joins in c.layer_runs()])
