"""Builder of the Sazepel decoder from ``SazepelConfig``: which parts stand in which layer, with which constants and
tensor names.

Embedding ``embed`` under a norm ``embed.norm``.  Per layer ``l<i>`` a `SandwichBlock`: a norm in front of and behind each
branch (``l<i>.norm1``, ``l<i>.norm1b``, ``l<i>.norm2``, ``l<i>.norm2b``); these norms, the embedding's and ``final.norm``
have ONE number as their weight.  The mixer, by ``type``:

* ``retention``: a `DecayedLinearAttention` in its retention form (``l<i>.mix.{q,k,v,g,o}``), rotated by half-split pairs,
  whose matrix state lives in the request's state slot;
* ``parallel``: `ParallelMixers` of a `PagedAttention` with talking heads (``l<i>.mix.left.{q,k,v,g,talk,o}``: unit-norm
  queries, keys and values without rotation, a gate element by element) and such a retention (``l<i>.mix.right.*``), the
  outputs normed (``l<i>.mix.left.out``, ``l<i>.mix.right.out``) and averaged.

The feed-forward, unless ``mlp`` is null: `RoutedExperts` (``l<i>.mlp.e<k>.{gate,up,down}``) whose router
(``l<i>.mlp.router``, ``l<i>.mlp.router.b``) weighs the chosen experts' outputs by a softmax over the chosen logits.
``final.norm``, ``head``, the logits times a constant.
"""

from __future__ import annotations

from slipstream_b200.config.sazepel_config import RetentionConfig, SazepelConfig
from slipstream_b200.parts import (DecayedLinearAttention, JoiningNorm, LMHead, NoPositionEncoding, PagedAttention,
                                   ParallelMixers, RotaryEncoding, RoutedExperts, SandwichBlock, TokenEmbedding)

from .decoder import DecoderLM

PAIR_SCALE = 0.5  # the result of two mixers side by side is the mean of their normed outputs


def build_sazepel(config: SazepelConfig) -> DecoderLM:
    c = config
    width = c.hidden_size
    blocks, rotaries = [], {}

    def norm(tensor: str) -> JoiningNorm:
        return JoiningNorm(tensor, width, c.norm_eps, scalar=True)

    def retention(name: str, m: RetentionConfig) -> DecayedLinearAttention:
        rotary = None
        if m.rot is not None:  # one table per distinct rotation
            key = (m.rot, m.dim)
            if key not in rotaries:
                rotaries[key] = RotaryEncoding(m.dim, m.rot.base, m.rot.dims, exact_table=True)
            rotary = rotaries[key]
        return DecayedLinearAttention(name, width, m.heads, m.dim, m.vdim, m.decay, c.norm_eps, retention=True,
                                      position_encoding=rotary)

    for i, layer in enumerate(c.layers):
        p, m = f"l{i}", layer.mixer
        if layer.type == "retention":
            mixer = retention(f"{p}.mix", m)
        else:
            a = m.left
            left = PagedAttention(f"{p}.mix.left", width, a.heads, a.kv_heads, a.dim, NoPositionEncoding(), qkv_bias=False,
                                  scale=a.scale, value_dim=a.vdim, unit_norm_eps=c.norm_eps, value_norm_eps=c.norm_eps,
                                  gate=True, talk=True, names={r: f"{p}.mix.left.{r}" for r in ("q", "k", "v", "g", "o", "talk")})
            mixer = ParallelMixers(left, retention(f"{p}.mix.right", m.right), PAIR_SCALE, PAIR_SCALE,
                                   out_norms=(f"{p}.mix.left.out", f"{p}.mix.right.out", c.norm_eps), hidden_size=width)
        ffn = None
        if layer.mlp is not None:
            f = layer.mlp
            ffn = RoutedExperts(f"{p}.mlp", width, f.ff, f.experts, f.top, renormalize=True, weight_on_input=False,
                                scores="softmax", router_tensor=f"{p}.mlp.router", router_bias=f"{p}.mlp.router.b",
                                expert_names=f"{p}.mlp.e{{e}}.{{role}}")
        blocks.append(SandwichBlock(mixer, ffn, norm(f"{p}.norm1"), norm(f"{p}.norm1b"),
                                    norm(f"{p}.norm2") if ffn is not None else None,
                                    norm(f"{p}.norm2b") if ffn is not None else None))
    return DecoderLM(
        c,
        TokenEmbedding("embed", c.vocab_size, width, tensor="embed", norm=norm("embed.norm")),
        blocks,
        norm("final.norm"),
        LMHead("head", c.vocab_size, width, tied_to=None, tensor="head", scale=c.logit_scale))
